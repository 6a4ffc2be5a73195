"""Somopel on the GPU against the plain restatement in somopel_oracle.py: every mechanism alone, prompts, portions, decoding, chunk
edges, far keys, steep and flat decays, odd sizes, re-used sequences, operators, and generation through the session layer."""
import copy
import io
import json

import numpy as np
import pytest

import somopel_oracle as so
from kmll_b200 import registry, somopel, trace
from kmll_b200 import runtime as rt
from kmll_b200.checkpoint import write_safetensors
from kmll_b200.lib import KmllError, load
from kmll_b200.session import GenerationOptions, SamplingOptions, Session

pytestmark = pytest.mark.gpu

# relative to the root mean square of the logits (or of the residual stream), per position; bf16: activations of the projections
TOL = {"float32": 5e-5, "bfloat16": 4e-2}
DTYPES = ["float32", "bfloat16"]


def parallel(heads=4, kv_heads=2, dim=16, vdim=24, size=19, scale=0.3, rheads=3, rdim=20, rvdim=16, tau=8.0, left=0.8, right=1.3, ff=None):
    return {"type": "parallel", "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": size}},
                                          "left_scale": left, "right": {"heads": rheads, "dim": rdim, "vdim": rvdim, "tau": tau}, "right_scale": right},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def delta(heads=4, kv_heads=2, dim=12, vdim=20, conv=4, ff=None):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(layers, width=72, vocab=130, positions=512, eps=1e-5, scale=2.5, logits=0.7):
    return {"architecture": "Somopel", "width": width, "vocab": vocab, "max_positions": positions, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "logit_scale": logits, "layers": copy.deepcopy(layers)}


MIXED = [parallel(ff=100), delta(ff=88), parallel(heads=3, kv_heads=3, size=70, rheads=2, rdim=16, rvdim=28), delta(heads=2, kv_heads=2, conv=3)]


def bits(a):
    return (np.ascontiguousarray(a, dtype=np.float32).view(np.uint32) >> 16).astype(np.uint16)


class Model:
    def __init__(self, cfg, dtype, seed=0, tensors=None, max_seq_len=None, ranks=None, edit=None):
        self.cfg, self.dtype = cfg, dtype
        self.tensors = so.random_tensors(cfg, seed, ranks=ranks) if tensors is None else tensors
        if edit is not None:
            edit(self.tensors)
        self.tensors = {n: so.bf16_round(a) for n, a in self.tensors.items()}
        layered = somopel.layered_config(cfg, lambda n: self.tensors[n].shape, max_seq_len, dtype == "float32")
        self.dec = rt.LayeredDecoder(layered)
        for name, layer, tensor in somopel.tensor_names(cfg):
            self.dec.set_tensor(layer, tensor, bits(self.tensors[name]))

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
        return so.forward(self.cfg, self.tensors, tokens, **kw)

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
def set_to(suffix, value, spread=0.3):
    def edit(T):
        rng = np.random.default_rng(77)
        for n in T:
            if n.endswith(suffix):
                T[n] = np.asarray(value + spread * rng.standard_normal(T[n].shape), dtype=np.float32)
    return edit


ALONE = {"attention": (parallel(right=0.0), None), "attention_one_group": (parallel(heads=20, kv_heads=1, dim=8, vdim=8, right=0.0), None),
         "attention_no_groups": (parallel(heads=3, kv_heads=3, size=512, right=0.0), None), "attention_chunk_1": (parallel(size=1, right=0.0), None),
         "gated": (parallel(left=0.0), None), "gated_tau_1": (parallel(left=0.0, tau=1.0), None),
         "gated_flat": (parallel(left=0.0, tau=40.0), set_to("a2.b", 8.0)), "gated_steep": (parallel(left=0.0, tau=1.0), set_to("a2.b", -9.0, 6.0)),
         "delta": (delta(), None), "delta_conv_1": (delta(conv=1), None), "delta_conv_2": (delta(conv=2), None), "delta_conv_7": (delta(conv=7), None),
         "delta_one_key_head": (delta(heads=6, kv_heads=1, dim=10), None), "delta_own_keys": (delta(heads=3, kv_heads=3, vdim=36), None),
         "delta_flat": (delta(), set_to("A_log", -9.0)), "delta_steep": (delta(), set_to("A_log", 2.5, 1.5)), "delta_gone": (delta(), set_to("A_log", 12.0))}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(ALONE))
def test_mixer_alone(cuda, name, dtype):
    layer, edit = ALONE[name]
    m = Model(config([layer]), dtype, seed=5, edit=edit)
    tokens = m.tokens(150)  # three chunks of the prompt form
    want = m.oracle(tokens)
    check(m.run(tokens), want, dtype)
    check(m.run(tokens[:40], [1] * 40), want[:40], dtype)  # from the first token on, one by one
    check(m.run(tokens, [70] + [1] * 20 + [60]), want, dtype)
    off = copy.deepcopy(m.tensors)
    off["l0.mix.left.o" if "attention" in name else "l0.mix.right.o" if "gated" in name else "l0.mix.o"][:] = 0
    assert rel(so.forward(m.cfg, off, tokens), want).max() > 3 * TOL["bfloat16"]  # the mixer shows in the logits
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_feed_forward_norms_positions_and_scales_alone(cuda, dtype):
    cfg = config([parallel(left=0.0, right=0.0, ff=200)], width=64, eps=3e-2)  # the mixers add nothing; eps large enough to be seen
    m = Model(cfg, dtype, seed=2)
    tokens = m.tokens(20)
    per = []
    want = m.oracle(tokens, per_layer=per)
    check(m.run(tokens), want, dtype)
    check(m.run(tokens, [1] * 20), want, dtype)
    m.dec.reset()
    check(m.dec.layer_residuals(tokens)[0], per[0], dtype)
    for changed in ("pos", "embed.norm", "embed.norm.b", "l0.norm2", "l0.norm2.b", "final.norm", "final.norm.b", "l0.mlp.gate"):  # each of them shows
        T2 = {**m.tensors, changed: np.zeros_like(m.tensors[changed])}
        assert rel(so.forward(cfg, T2, tokens), want).max() > 3 * TOL["bfloat16"], changed
    for changed in ("embedding", "logit_scale", "norm"):
        c2 = copy.deepcopy(cfg)
        c2[changed] = {"embedding": {"scale": 1.0}, "logit_scale": 1.0, "norm": {"eps": 0.3}}[changed]
        assert rel(so.forward(c2, m.tensors, tokens), want).max() > TOL["bfloat16"], changed
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_residual_stream_layer_by_layer(cuda, dtype):
    m = Model(config(MIXED), dtype, seed=3)
    tokens = m.tokens(75)
    per = []
    m.oracle(tokens, per_layer=per)
    m.dec.reset()
    first, rest = m.dec.layer_residuals(tokens[:33]), m.dec.layer_residuals(tokens[33:])
    for l, want in enumerate(per):
        check(np.concatenate([first[l], rest[l]]), want, dtype)
    m.close()


# ---- prompts, portions, decoding ---------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [[200], [2], [3, 64, 1, 5], [63, 2, 65], [64], [70, 1, 1, 2], [199, 1], [4, 3]])
def test_cuts_do_not_matter(cuda, dtype, sizes):
    m = Model(config(MIXED), dtype, seed=7)
    tokens = m.tokens(200)
    check(m.run(tokens, parts(200, sizes)), m.oracle(tokens), dtype)
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_and_first_tokens(cuda, dtype):
    m = Model(config(MIXED), dtype, seed=8)
    tokens = m.tokens(330)
    want = m.oracle(tokens)
    check(m.run(tokens, [5] + [1] * 325), want, dtype)
    for n in (1, 2, 3, 4, 5):  # the convolutions reach before the start
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
        alone[name] = fresh.run(t, parts(len(t), [20, 1, 2]))
        fresh.close()
    for _ in range(2):
        np.testing.assert_array_equal(m.run(a, parts(150, [20, 1, 2])), alone["a"])
        np.testing.assert_array_equal(m.run(b, parts(37, [20, 1, 2])), alone["b"])
    m.close()


def test_prompt_longer_than_one_pass(cuda):
    cfg = config([parallel(heads=2, kv_heads=1, size=300, rheads=1, ff=32), delta(heads=1, kv_heads=1)], width=32, vocab=64, positions=4600)
    m = Model(cfg, "bfloat16", seed=4)
    tokens = m.tokens(4400)
    whole = m.run(tokens)
    check(m.run(tokens, parts(4400, [997, 64, 1])), whole.astype(np.float64), "bfloat16")
    m.close()


# ---- other sizes ---------------------------------------------------------------------------------------------------------------
ODD = {"odd": (config([parallel(heads=10, kv_heads=5, dim=9, vdim=11, size=23, rheads=3, rdim=13, rvdim=7, ff=37), delta(heads=6, kv_heads=3, dim=11, vdim=13, conv=5, ff=51),
                       delta(heads=5, kv_heads=1, dim=7, vdim=9)], width=51, vocab=77), 140, {"a1": 3, "g1": 13, "right.a1": 9}),
       "ones": (config([parallel(heads=1, kv_heads=1, dim=1, vdim=1, size=2, rheads=1, rdim=1, rvdim=1, tau=1.0, ff=1), delta(heads=1, kv_heads=1, dim=1, vdim=1, conv=1, ff=2)],
                       width=9, vocab=5), 70, {"a1": 1, "g1": 1, "right.a1": 1}),
       "wide_heads": (config([parallel(heads=6, kv_heads=2, dim=128, vdim=128, size=90, scale=0.09, rheads=2, rdim=128, rvdim=96),
                              delta(heads=2, kv_heads=1, dim=100, vdim=130)], width=256), 150, {"a1": 70, "g1": 48, "right.a1": 24}),
       "large_ranks": (config([parallel(rdim=64, rvdim=64), delta(dim=48, vdim=40)], width=96), 130, {"a1": 200, "g1": 136, "right.a1": 260}),
       "long_values": (config([parallel(heads=2, kv_heads=1, dim=72, vdim=200, size=77, rheads=1, rdim=24, rvdim=170), delta(heads=1, kv_heads=1, dim=72, vdim=160)], width=64), 130, None),
       "beyond_the_fast_forms": (config([parallel(heads=2, kv_heads=1, dim=280, vdim=300, size=33, scale=0.06, rheads=1, rdim=150, rvdim=24),
                                         delta(heads=2, kv_heads=1, dim=200, vdim=36, conv=9)], width=64), 80, None)}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(ODD))
def test_other_sizes(cuda, name, dtype):
    cfg, n, ranks = ODD[name]
    m = Model(cfg, dtype, seed=11, ranks=ranks)
    tokens = m.tokens(n)
    want = m.oracle(tokens)
    factor = 3.0 if name == "ones" else 1.5  # (one-wide heads put a root mean square over a single value on everything)
    check(m.run(tokens), want, dtype, factor)
    check(m.run(tokens, parts(n, [31, 2, 1, 1])), want, dtype, factor)
    m.close()


# ---- one key that stands out ---------------------------------------------------------------------------------------------------
MARK, ASK = 1, 2  # token MARK leaves a key that token ASK looks for


def beacon(layer, gain, width=96, vocab=60, positions=512):
    """A one-layer model whose token MARK leaves a value that token ASK picks up: both embeddings are axes of their own, ASK's
    query points along MARK's key.  No position vectors, so the pair means the same everywhere."""
    cfg = config([layer], width=width, vocab=vocab, positions=positions, scale=1.0, logits=1.0)
    T = so.random_tensors(cfg, 21)
    T["pos"][:] = 0.0
    for n in T:
        if n.endswith("norm1") or n == "embed.norm":
            T[n][:] = 1.0
        if n.endswith("norm1.b") or n == "embed.norm.b":
            T[n][:] = 0.0
    T["embed"][:, :2] = 0.0
    T["embed"][[MARK, ASK]] = 0.0
    for t, i in ((MARK, 0), (ASK, 1)):
        T["embed"][t, i] = np.sqrt(width)
    one, zero = np.ones(width), np.zeros(width)

    def seen(t):  # what the mixer reads for token t
        return so.layer_norm(so.layer_norm(T["embed"][t].astype(np.float64), one, zero, 1e-5), one, zero, 1e-5)

    mark, ask = seen(MARK), seen(ASK)
    m = layer["mixer"]
    if layer["type"] == "parallel" and m["right_scale"] == 0.0:
        a = m["left"]
        key = (T["l0.mix.left.k"] @ mark).reshape(a["kv_heads"], a["dim"])
        q = T["l0.mix.left.q"].reshape(a["heads"], a["dim"], width)
        q[:] = 0.0
        for h in range(a["heads"]):
            k = key[h // (a["heads"] // a["kv_heads"])]
            q[h, :, 1] = gain * k / (ask[1] * a["scale"] * (k @ k))  # score of the pair = gain
    elif layer["type"] == "parallel":
        T["l0.mix.right.k"][:, 0] *= 12.0  # a strong key
        T["l0.mix.right.q"][:] *= 0.1
        T["l0.mix.right.q"][:, 1] = gain * (T["l0.mix.right.k"] @ mark) / ask[1]
        T["l0.mix.right.a2"][:] = 0.0
        T["l0.mix.right.a2.b"][:] = 12.0  # next to no decay
    else:
        d = m["dim"]
        k = T["l0.mix.k"].reshape(m["kv_heads"], d, width)
        q = T["l0.mix.q"].reshape(m["kv_heads"], d, width)
        k[:, d // 2:, 0] = 0.0     # MARK's key lies in the first half of the channels, all others in the second
        k[:, :d // 2] = 0.0
        k[:, :d // 2, 0] = 0.3 * np.abs(np.random.default_rng(3).standard_normal((m["kv_heads"], d // 2))) + 0.1
        q[:] = 0.0
        q[:, :d // 2, 1] = 3 * gain * k[:, :d // 2, 0]
        for n in "qkv":
            T[f"l0.mix.{n}.conv"][:] = 0.0
            T[f"l0.mix.{n}.conv"][:, -1] = 1.0
        T["l0.mix.A_log"][:] = -12.0
        T["l0.mix.b"][:, 0] = 1.0  # MARK writes at full strength
        T["l0.mix.o"] *= 3.0
    return cfg, {n: so.bf16_round(a) for n, a in T.items()}


def placed(n, marks, asks, vocab=60, seed=5):
    t = np.random.default_rng(seed).integers(3, vocab, n)
    t[list(marks)] = MARK
    t[list(asks)] = ASK
    return t


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size", [2, 7, 16, 64, 65, 100, 129])
def test_chunk_edges(cuda, dtype, size):
    cfg, T = beacon(parallel(heads=4, kv_heads=2, dim=16, vdim=24, size=size, right=0.0), 9.0)
    m = Model(cfg, dtype, tensors=T)
    # the last position of a chunk just sees a mark at its first; the first of the next chunk just misses one right ahead of it
    start = size * (1 + 40 // size)
    n = start + 2 * size + 3
    inside = placed(n, [start], [start + size - 1])
    outside = placed(n, [start + size - 1], [start + size])
    for tokens, at, wrong in ((inside, start + size - 1, size - 1), (outside, start + size, size + 1)):
        want = m.oracle(tokens)
        off = copy.deepcopy(cfg)
        off["layers"][0]["mixer"]["left"]["mask"]["size"] = wrong
        far = copy.deepcopy(cfg)
        far["layers"][0]["mixer"]["left"]["mask"]["size"] = 10 ** 6
        seen = [rel(so.forward(c, m.tensors, tokens), want) for c in (off, far)]
        assert max(s.max() for s in seen) > 5 * TOL["bfloat16"] and (tokens is inside or seen[1][at] > 5 * TOL["bfloat16"])
        check(m.run(tokens), want, dtype)                                             # in a prompt
        check(m.run(tokens, [start - 1] + [1] * (n - start + 1)), want, dtype)        # decoded
        check(m.run(tokens, [start - 1] + parts(n - start + 1, [2, 3])), want, dtype)  # in short portions
        check(m.run(tokens, [start + 1, size - 1, n - start - size]), want, dtype)    # portions end at the chunk's edges
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["gated", "delta"])
def test_far_keys_and_chunk_edges_of_the_recurrences(cuda, dtype, kind):
    layer = parallel(left=0.0, rheads=2, rdim=16, rvdim=24, tau=20.0) if kind == "gated" else delta(heads=4, kv_heads=2, dim=24, vdim=16)
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
def test_a_channel_that_forgets_within_a_chunk(cuda, dtype):
    """Some channels lose everything at single tokens and nothing in between: the running sums of the log decays jump."""
    cfg = config([parallel(left=0.0, rheads=2, rdim=24, rvdim=16, tau=1.0)])
    T = so.random_tensors(cfg, 31)
    T["l0.mix.right.a2"] *= 0.05
    T["l0.mix.right.a2.b"][:] = 9.0
    T["l0.mix.right.a1"][:, 0] = 40.0         # tokens with a large first entry drop the first half of the channels
    T["l0.mix.right.a2"].reshape(2, 24, -1)[:, :12] = -3.0
    T["embed"][:, 0] = 0.0
    T["embed"][::7, 0] = 3.0
    m = Model(cfg, dtype, tensors=T)
    tokens = m.tokens(140)
    want = m.oracle(tokens)
    check(m.run(tokens), want, dtype)
    check(m.run(tokens, parts(140, [50, 1, 30])), want, dtype)
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
    T = so.random_tensors(cfg, 14)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    write_safetensors(str(tmp_path / "model.safetensors"), {n: bits(a) for n, a in T.items()})
    return str(tmp_path), cfg, T


@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation(cuda, model_dir, dtype):
    path, cfg, T = model_dir
    s = Session(registry.load_model(path, dtype, max_seq_len=160))
    prompt = np.random.default_rng(6).integers(0, cfg["vocab"], 45)
    res = s.run_generation_request(prompt, GenerationOptions(max_new_tokens=40))
    gen = res["generated_tokens"]
    assert len(gen) == 40 and res["finish_reason"] == ("max-new-tokens", None) and res["backend"].startswith("bf16")
    want = so.forward(cfg, T, np.concatenate([prompt, gen]))  # the oracle, fed the same tokens, prefers each of them
    scale = np.sqrt((want * want).mean())
    for i, t in enumerate(gen):
        row = want[len(prompt) + i - 1]
        assert row.max() - row[t] <= 6 * TOL[dtype] * scale, i
    stop = gen[17]
    first = gen.index(stop)
    for chunk in (16, 7, 1):  # a stop token ends the run whatever the size of the device-resident chunks
        s.CHUNK = chunk
        s.prefill(prompt)
        assert [x.token_id for x in s.generate_greedy_until(40, 1, stop)] == gen[:first + 1]
        assert [x.token_id for x in s.generate_greedy_until(5)] == gen[first + 1:first + 6]
    s.prefill(prompt)
    assert [x.token_id for x in s.generate_sampled_top_k_until(8, 4, None, SamplingOptions(temperature=0.0))] == gen[:8]
    logits = s.next_logits_to_host()
    assert rel(logits[None].astype(np.float64), want[len(prompt) + 7][None]).max() <= 2 * TOL[dtype]
    s.reset_sequence()
    s.extend(prompt[:20])
    s.extend(prompt[20:])
    assert [x.token_id for x in s.generate_greedy_until(10)] == gen[:10]
    with pytest.raises(KmllError):
        s.run_generation_request(prompt, GenerationOptions(max_new_tokens=200))
    s.dec.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_replayed_requests_of_unequal_length(cuda, model_dir, tmp_path, dtype):
    path, cfg, T = model_dir
    rng = np.random.default_rng(8)
    requests = {name: rng.integers(0, cfg["vocab"], n) for name, n in (("a", 90), ("b", 1), ("c", 33), ("d", 7))}
    cuts = {"a": [64, 1, 2, 23], "b": [1], "c": [2, 1, 30], "d": [7]}
    lines, want, step = [], {}, 0
    for name, tokens in requests.items():
        full, at = so.forward(cfg, T, tokens), 0
        for n in cuts[name]:
            lines.append(json.dumps({"step": step, "entries": [{"id": name, "tokens": tokens[at:at + n].tolist(), "want": [n - 1]}],
                                     "end": [name] if at + n == len(tokens) else []}))
            want[step] = full[at + n - 1]
            at, step = at + n, step + 1
    s, out = Session(registry.load_model(path, dtype)), io.StringIO()
    trace.replay(s, lines, str(tmp_path), out)
    assert out.getvalue().split() == [w for i in range(step) for w in ("done", str(i))]
    for i, row in want.items():
        check(np.fromfile(tmp_path / f"{i}.f32", "<f4")[None], row[None], dtype, 1.5)
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
        check(m.dec.extend(seq[position:position + 5], range(5)), want[position:position + 5], "float32")
        m.dec.prefill(tokens)
        m.dec.generate_greedy(20)
    m.close()


def test_limits_and_tensors(cuda):
    m = Model(config([parallel(ff=24), delta()], positions=40), "bfloat16")
    with pytest.raises(KmllError):
        m.dec.extend(m.tokens(41))
    with pytest.raises(KmllError):
        rt.BatchDecoder(m.dec, 2)
    m.dec.reset()
    assert m.dec.extend(m.tokens(40), [39]).shape == (1, m.cfg["vocab"])
    with pytest.raises(KmllError):
        m.dec.extend([1])
    for name, layer, tensor in somopel.tensor_names(m.cfg):  # every tensor reads back, also the interleaved and the concatenated ones
        np.testing.assert_array_equal(m.dec.get_tensor(layer, tensor), bits(m.tensors[name]), err_msg=name)
    with pytest.raises(KmllError):
        m.dec.set_tensor(1, rt.T_W1, np.zeros((1, 1), np.uint16))
    fresh = rt.LayeredDecoder(m.dec.cfg)
    with pytest.raises(KmllError):
        fresh.extend([1])  # no weights
    assert load().kmll_decoder_init_random(fresh._h, 3, 0.05, 1) == 0
    assert np.isfinite(fresh.extend(m.tokens(20), [19])).all() and np.isfinite(fresh.extend([3], [0])).all()
    fresh.close()
    m.close()


# ---- operators through the C ABI --------------------------------------------------------------------------------------------
def test_linear_operators(cuda):
    import torch

    from kmll_b200 import ops
    gen = torch.Generator(device="cuda").manual_seed(9)

    def randn(*shape):
        return torch.randn(shape, generator=gen, device="cuda")

    def f64(t):
        return t.double().cpu().numpy()

    ws = ops.linear_batched_bf16_workspace()
    for batch, rows, cols in ((1, 6, 8), (3, 130, 72), (40, 1000, 2056), (64, 128, 4096), (300, 1300, 320)):
        w, x = (randn(rows, cols) / cols ** 0.5).bfloat16(), randn(batch, cols) * 2 + 0.5
        nw, nb = randn(cols).bfloat16(), randn(cols).bfloat16()
        W, X = f64(w), f64(x)
        want = so.gelu_tanh(f64(x.bfloat16()) @ W[0::2].T) * (f64(x.bfloat16()) @ W[1::2].T)
        for workspace in (None, ws):
            np.testing.assert_allclose(f64(ops.pair_linear_batched_bf16(x.bfloat16(), w, rt.ACT_GELU_TANH, workspace=workspace)), want, atol=0.1, rtol=0.01)
        want = so.gelu_tanh(X @ W[0::2].T) * (X @ W[1::2].T)
        np.testing.assert_allclose(f64(ops.pair_linear_batched_bf16(x, w, rt.ACT_GELU_TANH)), want, atol=1e-4, rtol=1e-4)
        n = so.layer_norm(X[0], f64(nw), f64(nb), 1e-3)
        np.testing.assert_allclose(f64(ops.normed_linear_bf16(x[0].contiguous(), w, rt.NORM_LAYER, nw, nb, 1e-3, out_scale=0.3)), 0.3 * (W @ n), atol=2e-5 * cols ** 0.5)
        got = ops.normed_linear_bf16(x[0].contiguous(), w, rt.NORM_LAYER, nw, nb, 1e-3, pair_act=rt.ACT_SILU)
        np.testing.assert_allclose(f64(got), so.silu(W[0::2] @ n) * (W[1::2] @ n), atol=1e-4 * cols ** 0.5)
        np.testing.assert_allclose(f64(ops.norm_rows_bf16(x, rt.NORM_LAYER, nw, nb, 1e-3)), so.layer_norm(X, f64(nw), f64(nb), 1e-3), atol=2e-2, rtol=1e-2)
    att = rt.MixerSpec(rt.MIXER_ATTENTION, 3, 4, 7, gate_act=rt.ACT_SIGMOID, out_scale=0.6)  # 21 columns, three of padding
    lin = rt.MixerSpec(rt.MIXER_GATED_LINEAR, 2, 4, 9, gate_act=rt.ACT_SILU, out_scale=1.7, out_norm=rt.OUT_NORM_HEAD_WEIGHTED)
    o, g0, g1, hw, res = randn(24 + 18), randn(3), randn(18), randn(9).bfloat16(), randn(50)
    o[21:24] = float("nan")  # the padding is never read as a number
    w = torch.zeros((50, 48), device="cuda", dtype=torch.bfloat16)
    w[:, :42] = randn(50, 42).bfloat16()
    O = f64(o)
    z = np.zeros(48)
    z[:21] = 0.6 * (O[:21].reshape(3, 7) * so.sigmoid(f64(g0))[:, None]).reshape(-1)
    z[24:42] = 1.7 * (so.rms(O[24:].reshape(2, 9), 1e-3) * f64(hw)).reshape(-1) * so.silu(f64(g1))
    from kmll_b200.lib import check as ok
    specs = (rt._MixerSpec * 2)(att._mixer(), lin._mixer())
    y = torch.empty(50, device="cuda")
    ok(load().kmll_mixer_output_linear_bf16(None, specs, 2, o.data_ptr(), ops._pointers([None, hw]), ops._pointers([g0, g1]), 1e-3, w.data_ptr(), 48, 50, 42,
                                            res.data_ptr(), y.data_ptr()))
    torch.cuda.synchronize()
    np.testing.assert_allclose(f64(y), f64(w) @ z + f64(res), atol=2e-5)


def test_attention_operator(cuda):
    import torch

    from kmll_b200 import ops
    gen = torch.Generator(device="cuda").manual_seed(10)
    for H, G, d, v, size, window, n in ((6, 2, 24, 16, 50, 0, 170), (4, 4, 64, 64, 0, 0, 300), (17, 1, 128, 128, 0, 37, 90), (8, 2, 200, 250, 33, 0, 70), (4, 1, 40, 136, 0, 0, 1100)):
        m = rt.MixerSpec(rt.MIXER_ATTENTION, H, d, v, kv_heads=G, score_scale=2.0 * d ** -0.5, chunk=size, window=window)
        ld = (H + G) * d + G * v
        x = torch.randn((n, ld), generator=gen, device="cuda").bfloat16()
        X = x.double()
        q, k, vv = X[:, :H * d].view(n, H, d), X[:, H * d:(H + G) * d].view(n, G, d), X[:, (H + G) * d:].view(n, G, v)
        s = torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(H // G, 1)) * m.score_scale
        i, j = torch.arange(n, device="cuda")[:, None], torch.arange(n, device="cuda")[None]
        seen = j <= i
        if size:
            seen &= (i // size) == (j // size)
        if window:
            seen &= j > i - window
        want = torch.einsum("hij,jhd->ihd", torch.softmax(s.masked_fill(~seen, float("-inf")), -1), vv.repeat_interleave(H // G, 1)).reshape(n, H * v)
        pad = lambda c: (c + 7) // 8 * 8
        for f32, tol in ((False, 2e-5), (True, 2e-5)):
            cache = torch.zeros((n + 3, G * (pad(d) + pad(v))), dtype=torch.float32 if f32 else torch.bfloat16, device="cuda")
            xx = x.float() if f32 else x
            off = (0, H * d, (H + G) * d)
            half = n // 2 + 1
            got = torch.cat([ops.grouped_attention(m, xx[:half].contiguous(), off, 0, cache), ops.grouped_attention(m, xx[half:].contiguous(), off, half, cache)])
            assert float((got.double() - want).abs().max()) <= tol, (H, G, d, v, f32)
            for p in (n - 1, half, 0):  # one token over the rows in place
                at = torch.tensor([p, 0, 0, 0], dtype=torch.int32, device="cuda")
                got = ops.grouped_attention(m, x[p:p + 1].float().contiguous(), off, at, cache)
                assert float((got.double() - want[p]).abs().max()) <= tol, (H, G, d, v, f32, p)


def test_gated_linear_operator(cuda):
    import torch

    from kmll_b200 import ops
    gen = torch.Generator(device="cuda").manual_seed(11)

    def randn(*shape):
        return torch.randn(shape, generator=gen, device="cuda")

    def f64(t):
        return t.double().cpu().numpy()

    H, G, d, v, n, rank, taps = 4, 2, 40, 24, 150, 16, 4
    for delta_rule in (0, 1):
        m = rt.MixerSpec(rt.MIXER_GATED_LINEAR, H, d, v, kv_heads=G, q_scale=0.2, decay_kind=rt.DECAY_SOFTPLUS if delta_rule else rt.DECAY_LOGISTIC, decay_tau=3.0,
                         decay_rank=rank, delta=delta_rule, conv=taps if delta_rule else 0, unit_eps=1e-6 if delta_rule else 0.0, gate_rank=8 if delta_rule else 0)
        off = (0, G * d, 2 * G * d, 2 * G * d + H * v, 2 * G * d + H * v + rank + 8, 2 * G * d + H * v + rank)
        x = randn(n, off[4] + 8).bfloat16()
        up, bias, alog, conv, gup = randn(H * d, rank).bfloat16(), randn(H * d).bfloat16(), randn(H).bfloat16(), randn(2 * G * d + H * v, taps).bfloat16(), randn(H * v, 8).bfloat16()
        X = f64(x)
        raw = X[:, :off[3]]
        if delta_rule:
            raw = so.silu(so.short_convolution(raw, f64(conv)))
        q, k, vv = so.heads_first(raw[:, :G * d], G), so.heads_first(raw[:, G * d:2 * G * d], G), so.heads_first(raw[:, 2 * G * d:], H)
        z = so.heads_first(X[:, off[3]:off[3] + rank] @ f64(up).T + f64(bias), H)
        if delta_rule:
            g = np.exp(-np.exp(f64(alog))[:, None, None] * so.softplus(z))
            want = so.delta_rule(so.unit(q) * 0.2, so.unit(k), vv, g, so.sigmoid(X[:, off[4]:off[4] + H]))
        else:
            alpha = np.exp(so.log_sigmoid(z) / 3.0)
            want = so.decayed_linear_attention(np.repeat(q, H // G, 0) * 0.2, np.repeat(k, H // G, 0), vv, alpha)
        want = so.heads_last(want)
        scale = np.sqrt((want * want).mean())
        for cut in ([n], [64, 86], [1] * 10 + [70, 5, 2, 63]):
            state, ring, out, at = torch.zeros(H * d * v, device="cuda"), torch.zeros(taps * (2 * G * d + H * v), device="cuda"), [], 0
            scratch = ops.gated_linear_scratch(m, n)
            gate = torch.zeros((n, H * v), device="cuda")
            for c in cut:
                out.append(ops.gated_linear_attention(m, x[at:at + c].contiguous(), off, at, state, up, bias, alog, conv, ring, gup, gate, scratch if c >= 4 else None))
                at += c
            err = np.abs(f64(torch.cat(out)) - want).max() / scale
            assert err <= 2e-3, (delta_rule, cut, err)
        if delta_rule:
            ops.gated_linear_attention(m, x, off, 0, torch.zeros_like(state), up, bias, alog, conv, torch.zeros_like(ring), gup, gate)
            np.testing.assert_allclose(f64(gate), X[:, off[5]:off[5] + 8] @ f64(gup).T, atol=1e-4)
