"""Plain, slow restatement of the layered decoder in numpy: one function per mechanism, written from the equations, sharing
no code with the package.  Everything is evaluated in float64 on the values the model stores, token by token or row by row,
so it depends neither on chunking nor on a cache."""
from __future__ import annotations

import math

import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def rms(x, eps):
    """x over its root mean square along the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rms_norm_zero_centred(x, w, eps):
    return rms(x, eps) * (1.0 + w)


def rms_norm_plain(x, w, eps):
    return rms(x, eps) * w


def rope_inverse_frequencies(rot):
    """(frequencies[dims / 2], factor on cos and sin)."""
    dims, base = rot["dims"], rot["base"]
    f = np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)])
    s = rot.get("scaling")
    if not s:
        return f, 1.0

    def where(turns):
        return dims * math.log(s["original"] / (2 * math.pi * turns)) / (2 * math.log(base))

    lo = max(math.floor(where(s["fast"])), 0)
    hi = min(math.ceil(where(s["slow"])), dims - 1)
    ramp = np.array([min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(dims // 2)])
    return f / s["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(s["factor"]) + 1.0


def rotate(x, positions, rot):
    """x [..., tokens, d]: the first rot.dims entries are rotated, entry i with entry i + dims / 2."""
    f, m = rope_inverse_frequencies(rot)
    half = rot["dims"] // 2
    a = np.asarray(positions, dtype=np.float64)[:, None] * f[None, :]
    c, s = np.cos(a) * m, np.sin(a) * m
    y = np.array(x, dtype=np.float64)
    u, v = x[..., :half], x[..., half:2 * half]
    y[..., :half] = u * c - v * s
    y[..., half:2 * half] = v * c + u * s
    return y


def softmax(x):
    e = np.exp(x - np.max(x, axis=-1, keepdims=True))
    return e / np.sum(e, axis=-1, keepdims=True)


def heads_first(x, heads):
    """[tokens, heads * d] -> [heads, tokens, d]"""
    t = x.shape[0]
    return np.transpose(x.reshape(t, heads, -1), (1, 0, 2))


def heads_last(x):
    return np.transpose(x, (1, 0, 2)).reshape(x.shape[1], -1)


def latent_attention(h, w, m, eps):
    """h [tokens, width]; w: tensors by short name; m: the mixer's sizes.  Keys and values of every head are written out."""
    t = h.shape[0]
    H, d, r, R = m["heads"], m["dim"], m["rot_dim"], m["kv_rank"]
    pos = np.arange(t)
    q = heads_first(h @ w["q"].T, H)
    both = h @ w["dkv"].T
    c = rms_norm_plain(both[:, :R], w["dkv.norm"], eps)
    kr = rotate(both[:, R:], pos, m["rot"])
    k = heads_first(c @ w["uk"].T, H)
    v = heads_first(c @ w["uv"].T, H)
    qr = rotate(q[..., d:], pos, m["rot"])
    out = np.zeros((H, t, m["vdim"]))
    for i in range(t):
        lo = max(0, i - m["mask"]["size"] + 1)
        for n in range(H):
            s = (k[n, lo:i + 1] @ q[n, i, :d] + kr[lo:i + 1] @ qr[n, i]) * m["scale"]
            out[n, i] = softmax(s) @ v[n, lo:i + 1]
    return heads_last(out) @ w["o"].T


def linear_recurrence(q, k, v, decay):
    """[heads, tokens, d]: S <- decay S + k v^T, o = S^T q, one token after the other."""
    H, t, d = q.shape
    out = np.zeros((H, t, v.shape[2]))
    for n in range(H):
        S = np.zeros((d, v.shape[2]))
        for i in range(t):
            S = decay[n] * S + np.outer(k[n, i], v[n, i])
            out[n, i] = q[n, i] @ S
    return out


def retention(h, w, m, eps):
    pos = np.arange(h.shape[0])
    H = m["heads"]
    q = rotate(heads_first(h @ w["q"].T, H), pos, m["rot"])
    k = rotate(heads_first(h @ w["k"].T, H), pos, m["rot"]) / math.sqrt(m["dim"])
    v = heads_first(h @ w["v"].T, H)
    o = rms(linear_recurrence(q, k, v, m["decay"]), eps)
    return (heads_last(o) * silu(h @ w["g"].T)) @ w["o"].T


def lightning(h, w, m, eps):
    H = m["heads"]
    q, k, v = (heads_first(silu(h @ w[n].T), H) for n in "qkv")
    o = heads_last(linear_recurrence(q, k, v, m["decay"]))
    return (rms_norm_plain(o, w["norm"], eps) * sigmoid(h @ w["g"].T)) @ w["o"].T


def poly_norm(z, coef, eps):
    a, b, c, e = (float(x) for x in coef)
    return a * rms(z, eps) + b * rms(z ** 2, eps) + c * rms(z ** 3, eps) + e


def dense_feed_forward(h, w, eps):
    return poly_norm(h @ w["up"].T, w["act"], eps) @ w["down"].T


MIXERS = {"latent_attention": latent_attention, "retention": retention, "lightning": lightning}


def forward(config, tensors, tokens, per_layer=None):
    """Logits [tokens, vocab] of one sequence from position 0; the residual stream after every layer goes to per_layer."""
    eps = config["norm"]["eps"]
    T = {n: np.asarray(a, dtype=np.float64) for n, a in tensors.items()}
    tokens = np.asarray(tokens)
    x = T["embed"][tokens] + T["pos"][:len(tokens)]
    for i, layer in enumerate(config["layers"]):
        part = {p: {n[len(f"l{i}.{p}."):]: a for n, a in T.items() if n.startswith(f"l{i}.{p}.")} for p in ("mix", "mlp")}
        x = x + MIXERS[layer["type"]](rms_norm_zero_centred(x, T[f"l{i}.norm1"], eps), part["mix"], layer["mixer"], eps)
        if layer.get("mlp") is not None:
            x = x + dense_feed_forward(rms_norm_zero_centred(x, T[f"l{i}.norm2"], eps), part["mlp"], eps)
        if per_layer is not None:
            per_layer.append(x.copy())
    return rms_norm_zero_centred(x, T["final.norm"], eps) @ T["head"].T


# ---- small random models ----------------------------------------------------------------------------------------------
def bf16_round(x):
    u = np.ascontiguousarray(x, dtype=np.float32).view(np.uint32)
    return ((u + 0x7fff + ((u >> 16) & 1)) & np.uint32(0xffff0000)).view(np.float32)


def tensor_shapes(config):
    """name -> shape of every tensor of a model with this configuration."""
    w, out = config["width"], {}
    out["embed"], out["pos"] = (config["vocab"], w), (config["max_positions"], w)
    for i, layer in enumerate(config["layers"]):
        m, p = layer["mixer"], f"l{i}.mix."
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        out[f"l{i}.norm1"] = (w,)
        if layer["type"] == "latent_attention":
            r, R = m["rot_dim"], m["kv_rank"]
            out.update({p + "q": (H * (d + r), w), p + "dkv": (R + r, w), p + "dkv.norm": (R,), p + "uk": (H * d, R), p + "uv": (H * dv, R)})
        else:
            out.update({p + "q": (H * d, w), p + "k": (H * d, w), p + "v": (H * dv, w), p + "g": (H * dv, w)})
            if layer["type"] == "lightning":
                out[p + "norm"] = (H * dv,)
        out[p + "o"] = (w, H * dv)
        if layer.get("mlp") is not None:
            ff = layer["mlp"]["ff"]
            out.update({f"l{i}.norm2": (w,), f"l{i}.mlp.up": (ff, w), f"l{i}.mlp.down": (w, ff), f"l{i}.mlp.act": (4,)})
    out["final.norm"], out["head"] = (w,), (config["vocab"], w)
    return out


def random_tensors(config, seed, gain=1.0):
    """bf16-representable float32 weights: linear ~ N(0, gain / sqrt(in)), norms around their neutral value."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(config).items():
        if name.endswith(".act"):
            a = np.array([0.6, 0.3, 0.5, 0.05]) + 0.1 * rng.standard_normal(4)
        elif name.endswith("dkv.norm") or name.endswith("mix.norm"):
            a = 1.0 + 0.2 * rng.standard_normal(shape)
        elif len(shape) == 1:
            a = 0.2 * rng.standard_normal(shape)
        elif name in ("embed", "pos"):
            a = rng.standard_normal(shape) * (1.0 if name == "embed" else 0.3)
        else:
            a = rng.standard_normal(shape) * gain / math.sqrt(shape[1])
        out[name] = bf16_round(np.asarray(a))
    return out
