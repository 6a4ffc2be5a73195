"""Plain, slow restatement of the Somopel decoder in numpy (float64, token by token): one function per mechanism, written from
the equations, sharing no code with the package."""
from __future__ import annotations

import math

import numpy as np

from layered_oracle import bf16_round, heads_first, heads_last, rms, sigmoid, silu, softmax


def layer_norm(x, w, b, eps):
    d = x - np.mean(x, axis=-1, keepdims=True)
    return d / np.sqrt(np.mean(d * d, axis=-1, keepdims=True) + eps) * w + b


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus(z):
    return np.logaddexp(0.0, z)


def log_sigmoid(z):
    return -np.logaddexp(0.0, -z)


def embedding(T, tokens, scale, eps):
    x = T["embed"][tokens] * scale + T["pos"][:len(tokens)]
    return layer_norm(x, T["embed.norm"], T["embed.norm.b"], eps)


def chunked_attention(q, k, v, scale, size):
    """q [heads, tokens, dim], k / v [kv heads, tokens, ...]: a token sees the tokens of its own chunk up to itself."""
    H, t, _ = q.shape
    per = H // k.shape[0]
    out = np.zeros((H, t, v.shape[2]))
    for h in range(H):
        for i in range(t):
            lo = i // size * size
            s = k[h // per, lo:i + 1] @ q[h, i] * scale
            out[h, i] = softmax(s) @ v[h // per, lo:i + 1]
    return out


def decayed_linear_attention(q, k, v, alpha):
    """S <- diag(alpha) S + k v^T, o = S^T q; everything [heads, tokens, ...], alpha per key channel."""
    H, t, d = q.shape
    out = np.zeros((H, t, v.shape[2]))
    for h in range(H):
        S = np.zeros((d, v.shape[2]))
        for i in range(t):
            S = alpha[h, i][:, None] * S + np.outer(k[h, i], v[h, i])
            out[h, i] = S.T @ q[h, i]
    return out


def short_convolution(x, taps):
    """x [tokens, channels], taps [channels, n]: the last tap is the current token's."""
    t, n = x.shape[0], taps.shape[1]
    padded = np.concatenate([np.zeros((n - 1, x.shape[1])), x])
    return sum(padded[j:j + t] * taps[:, j] for j in range(n))


def unit(x):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


def delta_rule(q, k, v, g, beta):
    """S <- diag(g) S, u = beta (v - S^T k), S <- S + k u^T, o = S^T q; q and k per group of heads."""
    H, t, d = g.shape
    per = H // q.shape[0]
    out = np.zeros((H, t, v.shape[2]))
    for h in range(H):
        S = np.zeros((d, v.shape[2]))
        for i in range(t):
            kk = k[h // per, i]
            S = g[h, i][:, None] * S
            u = beta[i, h] * (v[h, i] - S.T @ kk)
            S = S + np.outer(kk, u)
            out[h, i] = S.T @ q[h // per, i]
    return out


def attention_half(h, w, m):
    H, G = m["heads"], m["kv_heads"]
    o = chunked_attention(heads_first(h @ w["q"].T, H), heads_first(h @ w["k"].T, G), heads_first(h @ w["v"].T, G), m["scale"], m["mask"]["size"])
    o = o * sigmoid(h @ w["g"].T).T[:, :, None]
    return heads_last(o) @ w["o"].T


def linear_half(h, w, m, eps):
    H = m["heads"]
    q = heads_first(h @ w["q"].T, H) / math.sqrt(m["dim"])
    k, v = heads_first(h @ w["k"].T, H), heads_first(h @ w["v"].T, H)
    alpha = np.exp(heads_first(log_sigmoid(h @ w["a1"].T @ w["a2"].T + w["a2.b"]) / m["tau"], H))
    o = rms(decayed_linear_attention(q, k, v, alpha), eps) * w["norm"]
    return (heads_last(o) * silu(h @ w["g"].T)) @ w["o"].T


def parallel(h, w, m, eps):
    half = {s: {n[len(s) + 1:]: a for n, a in w.items() if n.startswith(s + ".")} for s in ("left", "right")}
    return m["left_scale"] * attention_half(h, half["left"], m["left"]) + m["right_scale"] * linear_half(h, half["right"], m["right"], eps)


def channel_delta(h, w, m, eps):
    H, G = m["heads"], m["kv_heads"]
    q, k, v = (silu(short_convolution(h @ w[n].T, w[n + ".conv"])) for n in "qkv")
    q, k = unit(heads_first(q, G)) / math.sqrt(m["dim"]), unit(heads_first(k, G))
    g = heads_first(softplus(h @ w["a1"].T @ w["a2"].T + w["dt_bias"]), H)
    g = np.exp(-np.exp(w["A_log"])[:, None, None] * g)
    o = rms(delta_rule(q, k, heads_first(v, H), g, sigmoid(h @ w["b"].T)), eps) * w["norm"]
    return (heads_last(o) * sigmoid(h @ w["g1"].T @ w["g2"].T)) @ w["o"].T


def feed_forward(h, w):
    return (gelu_tanh(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


MIXERS = {"parallel": parallel, "channel_delta": channel_delta}


def forward(config, tensors, tokens, per_layer=None):
    """Logits [tokens, vocab] of one sequence from position 0; the residual stream after every layer goes to per_layer."""
    eps = config["norm"]["eps"]
    T = {n: np.asarray(a, dtype=np.float64) for n, a in tensors.items()}
    x = embedding(T, np.asarray(tokens), config["embedding"]["scale"], eps)
    for i, layer in enumerate(config["layers"]):
        part = {p: {n[len(f"l{i}.{p}."):]: a for n, a in T.items() if n.startswith(f"l{i}.{p}.")} for p in ("mix", "mlp")}
        h = layer_norm(x, T[f"l{i}.norm1"], T[f"l{i}.norm1.b"], eps)
        x = x + MIXERS[layer["type"]](h, part["mix"], layer["mixer"], eps)
        if layer.get("mlp") is not None:
            x = x + feed_forward(layer_norm(x, T[f"l{i}.norm2"], T[f"l{i}.norm2.b"], eps), part["mlp"])
        if per_layer is not None:
            per_layer.append(x.copy())
    return layer_norm(x, T["final.norm"], T["final.norm.b"], eps) @ T["embed"].T * config["logit_scale"]


# ---- small random models ----------------------------------------------------------------------------------------------
def tensor_shapes(config, ranks=None):
    """name -> shape of every tensor; `ranks`: inner sizes of the low-rank pairs (config.json does not name them)."""
    r = {"a1": 6, "g1": 10, "right.a1": 5, **(ranks or {})}
    w, out = config["width"], {}

    def norm(name):
        out[name], out[name + ".b"] = (w,), (w,)

    out["embed"], out["pos"] = (config["vocab"], w), (config["max_positions"], w)
    norm("embed.norm")
    for i, layer in enumerate(config["layers"]):
        m, p = layer["mixer"], f"l{i}.mix."
        norm(f"l{i}.norm1")
        if layer["type"] == "parallel":
            a, b = m["left"], m["right"]
            H, G = a["heads"], a["kv_heads"]
            out.update({p + "left.q": (H * a["dim"], w), p + "left.k": (G * a["dim"], w), p + "left.v": (G * a["vdim"], w), p + "left.g": (H, w),
                        p + "left.o": (w, H * a["vdim"])})
            K, V = b["heads"] * b["dim"], b["heads"] * b["vdim"]
            out.update({p + "right.q": (K, w), p + "right.k": (K, w), p + "right.v": (V, w), p + "right.g": (V, w), p + "right.o": (w, V),
                        p + "right.norm": (b["vdim"],), p + "right.a1": (r["right.a1"], w), p + "right.a2": (K, r["right.a1"]), p + "right.a2.b": (K,)})
        else:
            H, G, taps = m["heads"], m["kv_heads"], m["conv"]
            K, V = H * m["dim"], H * m["vdim"]
            for n, c in (("q", G * m["dim"]), ("k", G * m["dim"]), ("v", V)):
                out.update({p + n: (c, w), p + n + ".conv": (c, taps)})
            out.update({p + "b": (H, w), p + "A_log": (H,), p + "norm": (m["vdim"],), p + "a1": (r["a1"], w), p + "a2": (K, r["a1"]), p + "dt_bias": (K,),
                        p + "g1": (r["g1"], w), p + "g2": (V, r["g1"]), p + "o": (w, V)})
        if layer.get("mlp") is not None:
            norm(f"l{i}.norm2")
            ff = layer["mlp"]["ff"]
            out.update({f"l{i}.mlp.gate": (ff, w), f"l{i}.mlp.up": (ff, w), f"l{i}.mlp.down": (w, ff)})
    norm("final.norm")
    return out


def random_tensors(config, seed, gain=1.0, ranks=None):
    """bf16-representable float32 weights: linear ~ N(0, gain / sqrt(in)), norms around their neutral value."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(config, ranks).items():
        tail = name.rsplit(".", 1)[-1]
        z = rng.standard_normal(shape)
        if name in ("embed", "pos"):
            a = z * (0.5 if name == "embed" else 0.4)
        elif tail.startswith("norm"):
            a = 1.0 + 0.2 * z
        elif name.endswith("a2.b"):
            a = 2.0 + z
        elif tail == "dt_bias":
            a = -1.0 + z
        elif tail == "A_log":
            a = -0.5 + 0.7 * z
        elif tail == "conv":
            a = z * 0.6
        elif len(shape) == 1:
            a = 0.2 * z
        else:
            a = z * gain / math.sqrt(shape[1])
        out[name] = bf16_round(np.asarray(a))
    return out
