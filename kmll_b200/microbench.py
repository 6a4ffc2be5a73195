"""Kernel micro-benchmark: times one quantized linear operator shape inside a CUDA graph over several
distinct weight matrices (so every launch streams cold weights from HBM) and prints achieved GB/s.

  python -m kmll_b200.microbench --op silu_gate_up --fmt w4 --rows 14336 --cols 4096
  python -m kmll_b200.microbench --op linear --fmt i8 --rows 32000 --cols 4096 --mats 8 --reps 10

ops: linear, qkv (RMSNorm + Q/K/V), linear_residual, silu_gate_up (RMSNorm prologue on), linear_top1, attention (rows =
context length).  fmt: i8 (RS-I8), w4 (W4-G128 canonical layout), w4p (W4-G128 prepared layout).  --suite decode runs every
batch-1 operator shape of a Mistral-7B-architecture decode step.
"""
from __future__ import annotations

import argparse
import json
import os

import torch

from . import ops


def _weight(fmt, rows, cols):
    if fmt == "w4p":
        return ops.DeviceW4PMatrix.from_canonical(_weight("w4", rows, cols))
    if fmt == "w4":
        return ops.DeviceW4G128Matrix(torch.randint(0, 256, (rows, cols // 2), dtype=torch.uint8, device="cuda"),
                                      (torch.rand((rows, cols // 128), device="cuda") * 0.01 + 0.001).half(), rows, cols)
    return ops.DeviceRowwiseScaledI8Matrix(torch.randint(-127, 128, (rows, cols), dtype=torch.int8, device="cuda"),
                                           torch.rand(rows, device="cuda") * 0.01, rows, cols)


def weight_bytes(fmt, rows, cols):
    return rows * cols * 0.515625 if fmt in ("w4", "w4p") else rows * cols + 4 * rows


# the batch-1 operators of one Mistral-7B-architecture decode step: (op, rows, cols, distinct matrices)
DECODE_SUITE = [("qkv", 6144, 4096, 16), ("linear_residual", 4096, 4096, 16), ("silu_gate_up", 14336, 4096, 8),
                ("linear_residual", 4096, 14336, 8), ("linear_top1", 32000, 4096, 4)]


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--op", default="linear", choices=["linear", "qkv", "linear_residual", "silu_gate_up", "linear_top1", "attention", "linear_batched",
                                                        "decode_batch", "prefill"])
    ap.add_argument("--batch", type=int, default=16, help="rows of x for --op linear_batched (5..32: small-batch kernel; more: tcgen05 f16 kernel)")
    ap.add_argument("--fmt", default="w4", choices=["w4", "w4p", "i8"])
    ap.add_argument("--rows", type=int, default=14336)
    ap.add_argument("--cols", type=int, default=4096)
    ap.add_argument("--mats", type=int, default=8)
    ap.add_argument("--reps", type=int, default=10)
    ap.add_argument("--suite", default="", choices=["", "decode", "chain4096", "micro", "gemm_sweep", "layered", "somopel"],
                    help="layered: the kernels of the layered decoders beside their like kernels, and whole decoders; decode: every batch-1 operator shape of a Mistral-7B-architecture step; chain4096: 4096x4096 matvec + residual + "
                         "RMSNorm in both formats; micro: RMSNorm / SwiGLU / RoPE / row softmax over B in {1,16,64}, bf16; gemm_sweep: "
                         "M in {1,16,64,256,2048} x four (N,K), W4-G128")
    ap.add_argument("--only", default="", help="layered: only the lines of one part (matvec, mixer decode, gemm, mixer prompt, rows, decoder)")
    ap.add_argument("--shards", type=int, default=1, help="gemm_sweep: time one rank's share of every matrix when its N output rows are split over this "
                                                           "many GPUs (column-parallel: disjoint output blocks, no collective)")
    ap.add_argument("--profile", action="store_true", help="bracket one graph replay with cudaProfilerStart/Stop")
    ap.add_argument("--layers", type=int, default=2, help="decode_batch, prefill: layers of the Mistral-7B-shaped decoder (a small case for profiling)")
    ap.add_argument("--kv-bf16", action="store_true", help="decode_batch, prefill: keep the KV cache in bf16")
    a = ap.parse_args()
    torch.cuda.set_device(0)
    if a.suite == "decode":
        for op, rows, cols, mats in DECODE_SUITE:
            a.op, a.rows, a.cols, a.mats = op, rows, cols, mats
            run_one(a)
        return
    if a.suite == "chain4096":
        return suite_chain4096(a.reps)
    if a.suite == "micro":
        return suite_micro(a.reps)
    if a.suite == "gemm_sweep":
        return suite_gemm_sweep(a.reps, shards=a.shards)
    if a.suite == "layered":
        return suite_layered(a.reps, only=a.only)
    if a.suite == "somopel":
        return suite_somopel(a.reps, only=a.only)
    run_one(a)


def peak_hbm_gbs():
    path = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "MEASURED_PEAKS.json")
    try:
        with open(path) as f:
            p = json.load(f)
        return float(p["hbm_gbs"]), float(p["bf16_tflops"]), "measured"
    except (OSError, KeyError, ValueError):
        return 6650.0, 1590.0, "fallback"


def time_graph(calls, reps):
    """Average microseconds per call: the calls are captured once each in one CUDA graph, replayed `reps` times."""
    for c in calls[:2]:
        c()
    torch.cuda.synchronize()
    graph = torch.cuda.CUDAGraph()
    with torch.cuda.graph(graph):
        for c in calls:
            c()
    for _ in range(3):
        graph.replay()
    torch.cuda.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    for _ in range(reps):
        graph.replay()
    e1.record()
    torch.cuda.synchronize()
    return e0.elapsed_time(e1) * 1e3 / (reps * len(calls))


def report(name, us, alg_bytes, extra=None, flops=None, cpu_us=None):
    hbm, tf, src = peak_hbm_gbs()
    line = {"op": name, "us": round(us, 2), "algorithmic_mb": round(alg_bytes / 1e6, 3), "gbs": round(alg_bytes / us / 1e3, 1),
            "frac_hbm": round(alg_bytes / us / 1e3 / hbm, 3), "peak": src}
    if flops is not None:
        line["tflops"] = round(flops / us / 1e6, 1)
        line["frac_tensor"] = round(flops / us / 1e6 / tf, 3)
    if cpu_us is not None:
        line["cpu_us"] = round(cpu_us, 1)
        line["cpu_gbs"] = round(alg_bytes / cpu_us / 1e3, 2)
    if extra:
        line.update(extra)
    print(json.dumps(line), flush=True)


def suite_chain4096(reps, cpu=None):
    """y = dequant(W) x + r, h = RMSNorm(y): W 4096 x 4096 ~ N(0, 0.02) seed 0, x, r ~ N(0, 1), gamma ~ U(0.5, 1.5), eps 1e-6.
    `cpu(kind, **shape)`, when given, returns the microseconds a CPU implementation of the same operator takes."""
    rows = cols = 4096
    gen = torch.Generator(device="cuda").manual_seed(0)
    x = torch.randn(cols, generator=gen, device="cuda")
    r = torch.randn(rows, generator=gen, device="cuda")
    gamma = (torch.rand(rows, generator=gen, device="cuda") + 0.5).to(torch.bfloat16)
    y, h = torch.empty(rows, device="cuda"), torch.empty(rows, device="cuda")
    for fmt in ("i8", "w4", "w4p"):
        n = 24  # 24 distinct matrices: 200 to 400 MB, larger than L2
        calls = []
        for _ in range(n):
            w32 = torch.randn((rows, cols), generator=gen, device="cuda") * 0.02
            if fmt == "i8":
                w = ops.DeviceRowwiseScaledI8Matrix.from_bf16_rows_symmetric(ops.f32_to_bf16(w32))
            else:
                w = ops.DeviceW4G128Matrix.from_f32_rows(w32)
                if fmt == "w4p":
                    w = ops.DeviceW4PMatrix.from_canonical(w)
            calls.append(lambda w=w: (ops.linear_residual(x, w, r, out=y), ops.rmsnorm(y, gamma, 1e-6, out=h)))
        us = time_graph(calls, reps)
        alg = weight_bytes(fmt, rows, cols) + 4 * cols + 3 * 4 * rows + 2 * rows + 4 * rows
        report(f"matvec+residual then rmsnorm 4096x4096 [{fmt}] (2 launches)", us, alg,
               cpu_us=cpu("chain4096", fmt=fmt) if cpu else None)


def suite_micro(reps, cpu=None):
    """RMSNorm [B,4096], SwiGLU [B,11008], RoPE [B,32,128] theta 1e6 positions U[0,4096), row softmax [B*32,4096]; bf16, seed 1."""
    gen = torch.Generator(device="cuda").manual_seed(1)
    for B in (1, 16, 64):
        copies = max(2, int(300e6 // max(1, B * 32 * 4096 * 4)))  # distinct inputs so that together they exceed L2
        copies = min(copies, 64)

        def bf(*shape):
            return [torch.randn(shape, generator=gen, device="cuda").to(torch.bfloat16) for _ in range(copies)]

        xs, outs = bf(B, 4096), bf(B, 4096)
        gamma = (torch.rand(4096, generator=gen, device="cuda") + 0.5).to(torch.bfloat16)
        us = time_graph([lambda i=i: ops.rmsnorm_batched_bf16(xs[i], gamma, B, 4096, 1e-6, out=outs[i]) for i in range(copies)], reps)
        report(f"rmsnorm [{B},4096] bf16", us, B * 4096 * 4 + 2 * 4096, cpu_us=cpu("rmsnorm", batch=B) if cpu else None)
        g, u, o = bf(B, 11008), bf(B, 11008), bf(B, 11008)
        us = time_graph([lambda i=i: ops.silu_mul(g[i], u[i], out=o[i]) for i in range(copies)], reps)
        report(f"swiglu [{B},11008] bf16", us, 3 * B * 11008 * 2, cpu_us=cpu("swiglu", batch=B) if cpu else None)
        xr, orr = bf(B, 32, 128), bf(B, 32, 128)
        freqs = torch.tensor([1.0 / (1e6 ** (2 * i / 128)) for i in range(64)], dtype=torch.float32, device="cuda")
        pos = torch.randint(0, 4096, (B,), generator=gen, device="cuda", dtype=torch.int32)
        us = time_graph([lambda i=i: ops.apply_rope_batched_bf16(xr[i], freqs, pos, out=orr[i]) for i in range(copies)], reps)
        report(f"rope [{B},32,128] bf16", us, 2 * B * 32 * 128 * 2 + 4 * B, cpu_us=cpu("rope", batch=B) if cpu else None)
        sm_copies = max(2, min(copies, int(300e6 // (B * 32 * 4096 * 4))))
        sx = [torch.randn((B * 32, 4096), generator=gen, device="cuda").to(torch.bfloat16) for _ in range(sm_copies)]
        so = [torch.empty_like(t) for t in sx]
        us = time_graph([lambda i=i: ops.softmax_rows(sx[i], out=so[i]) for i in range(sm_copies)], reps)
        report(f"softmax [{B * 32},4096] bf16", us, 2 * B * 32 * 4096 * 2, cpu_us=cpu("softmax", batch=B) if cpu else None)


def suite_gemm_sweep(reps, cpu=None, shards=1):
    """Quantized GEMM sweep, W4-G128 (seed 4): M in {1, 16, 64, 256, 2048} x (N, K) in {(3584, 3584), (18944, 3584),
    (3584, 18944), (152064, 3584)}; activations are bf16-valued N(0, 1) held as f32 (the operator API is f32)."""
    gen = torch.Generator(device="cuda").manual_seed(4)
    for n_full, k in ((3584, 3584), (18944, 3584), (3584, 18944), (152064, 3584)):
        n = n_full // shards
        wbytes = n * k * 0.515625
        for m in (1, 16, 64, 256, 2048):
            mats = 1 if m >= 256 else max(1, min(48, int(300e6 // wbytes) + 1))
            ws = [_weight("w4", n, k) for _ in range(mats)]
            x = torch.randn((m, k), generator=gen, device="cuda").to(torch.bfloat16).float()
            out = torch.empty((m, n), device="cuda")
            if m == 1:
                if k <= 16384:
                    ws = [ops.DeviceW4PMatrix.from_canonical(w) for w in ws]
                calls = [lambda w=w: ops.linear(x[0], w, out=out[0]) for w in ws]
            else:
                scratch = ops.linear_batched_workspace(m, k)
                calls = [lambda w=w: ops.linear_batched(x, w, m, k, n, out=out, workspace=scratch) for w in ws]
            us = time_graph(calls, reps)
            report(f"gemm w4 M={m} N={n} K={k}", us, wbytes + 4 * m * k + 4 * m * n, flops=2.0 * m * n * k,
                   extra={"bound": "hbm" if m <= 16 else "tensor", "path": "stream kernel" if m == 1 else "tcgen05",
                          **({"shard_of": n_full, "shards": shards} if shards > 1 else {})},
                   cpu_us=cpu("gemm_w4", m=m, n=n, k=k) if cpu else None)
            del ws, calls
            torch.cuda.empty_cache()


# ---- layered decoders ---------------------------------------------------------------------------------------------------
# mixer sizes that resemble real layers of the given width
LAYERED_SIZES = {4096: dict(ff=14336, lightning=(32, 128, 128), retention=(16, 256, 256), latent=dict(heads=32, dim=128, rot=64, vdim=128, rank=512)),
                 2048: dict(ff=8192, lightning=(16, 128, 128), retention=(8, 256, 256), latent=dict(heads=16, dim=128, rot=64, vdim=128, rank=512))}
LAYERED_WINDOW = 4096


def layered_decoder(width, layers, max_seq_len, vocab=32000):
    """Random-weight decoder whose layers cycle through lightning, latent attention and retention."""
    from . import runtime as rt
    from .pefisun import layered_config
    z = LAYERED_SIZES[width]
    la = z["latent"]

    def layer(i):
        kind = ("lightning", "latent_attention", "retention")[i % 3]
        if kind == "latent_attention":
            m = {"heads": la["heads"], "dim": la["dim"], "rot_dim": la["rot"], "vdim": la["vdim"], "kv_rank": la["rank"], "scale": (la["dim"] + la["rot"]) ** -0.5,
                 "mask": {"size": LAYERED_WINDOW}, "rot": {"base": 1e4, "dims": la["rot"], "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}
        else:
            h, dk, dv = z["lightning" if kind == "lightning" else "retention"]
            m = {"heads": h, "dim": dk, "vdim": dv, "decay": [1.0 - 2.0 ** (-4 - 6 * j / h) for j in range(h)]}
            if kind == "retention":
                m["rot"] = {"base": 1e4, "dims": dk}
        return {"type": kind, "mixer": m, "mlp": {"kind": "dense", "ff": z["ff"]}}

    cfg = layered_config({"width": width, "vocab": vocab, "max_positions": max_seq_len, "norm": {"eps": 1e-5}, "layers": [layer(i) for i in range(layers)]})
    dec = rt.LayeredDecoder(cfg)
    dec.init_random(7, 0.02)
    return dec


def time_decoder(dec, prompt_len, steps, prefill_reps=3):
    """(decode ms per token at context prompt_len, prefill ms): CUDA events, after warm-up."""
    import numpy as np
    prompt = np.random.default_rng(3).integers(0, dec.cfg.vocab_size, prompt_len)
    dec.prefill(prompt)
    dec.prefill(prompt)
    e = [torch.cuda.Event(enable_timing=True) for _ in range(2)]
    best = None
    for _ in range(prefill_reps):
        torch.cuda.synchronize()
        e[0].record()
        dec.prefill(prompt)
        e[1].record()
        torch.cuda.synchronize()
        t = e[0].elapsed_time(e[1])
        best = t if best is None else min(best, t)
    dec.enqueue_steps(4)
    torch.cuda.synchronize()
    e[0].record()
    dec.enqueue_steps(steps)
    e[1].record()
    torch.cuda.synchronize()
    return e[0].elapsed_time(e[1]) / steps, best


def suite_layered(reps, cpu=None, only="", context=2048):
    """The kernels of the layered decoders beside the like kernels of the uniform decoder (RS-I8 and W4-G128 weights, f32 KV
    cache) at equal sizes, then whole decoders of equal width and layer count: decode at context 2048, 2048-token prompt.
    Inputs of a line together exceed L2.  frac_hbm / frac_tensor: of the copy bandwidth / bf16 peak."""
    from . import runtime as rt
    gen = torch.Generator(device="cuda").manual_seed(5)

    def bf(*shape, std=1.0):
        return (torch.randn(shape, generator=gen, device="cuda") * std).to(torch.bfloat16)

    def want(name):
        return not only or only in name

    def copies(nbytes):
        return max(2, min(48, int(300e6 // nbytes) + 1))

    n = context
    table = {r: torch.randn((n + 64, r // 2, 2), generator=gen, device="cuda") for r in (64, 256)}
    pos = torch.tensor([n, 0, 0, 0], dtype=torch.int32, device="cuda")
    for width, z in LAYERED_SIZES.items():
        ff, la = z["ff"], z["latent"]
        h, dk, dv = z["lightning"]
        rh, rdk, rdv = z["retention"]
        # ---- one row of x
        coef = bf(4)
        shapes = [("norm + stacked q k v gate", 2 * h * (dk + dv), width, "norm"), ("norm + up", ff, width, "norm"), ("polynorm + down", width, ff, "poly"),
                  ("gate + output projection", width, h * dv, "gate"), ("norm + lm_head", 32000, width, "norm")]
        for name, rows, cols, kind in shapes:
            if not want("matvec"):
                continue
            ws = [bf(rows, cols, std=0.02) for _ in range(copies(rows * cols * 2))]
            x, y, g, nw = torch.randn(cols, device="cuda"), torch.empty(rows, device="cuda"), torch.randn(cols, device="cuda"), bf(cols)
            res = torch.randn(rows, device="cuda")
            call = {"norm": lambda w: ops.linear_bf16(x, w, norm_weight=nw, norm_offset=1.0, eps=1e-5, out=y),
                    "poly": lambda w: ops.polynorm_linear_bf16(x, coef, 1e-5, w, residual=res, out=y),
                    "gate": lambda w: ops.gated_linear_bf16(x, g, w, 1e-5, head_len=dv, residual=res, out=y)}[kind]
            us = time_graph([lambda w=w: call(w) for w in ws], reps)
            report(f"matvec {name} {rows}x{cols} [bf16]", us, rows * cols * 2 + 4 * cols + 4 * rows)
            del ws
            for fmt in ("i8", "w4p"):
                ws = [_weight(fmt, rows, cols) for _ in range(copies(rows * cols // 2))]
                like = (lambda w: ops.linear_residual(x, w, res, out=y)) if kind != "norm" else (lambda w: ops.linear(x, w, out=y))
                us = time_graph([lambda w=w: like(w) for w in ws], reps)
                report(f"matvec {rows}x{cols} [{fmt}] (like kernel)", us, weight_bytes(fmt, rows, cols) + 4 * cols + 4 * rows)
                del ws
        # ---- mixers, one token
        if want("mixer decode"):
            for name, hh, d, v, rot in (("lightning", h, dk, dv, 0), ("retention", rh, rdk, rdv, rdk)):
                sb = hh * d * v * 4
                states = [torch.randn(hh * d * v, device="cuda") for _ in range(copies(2 * sb))]
                pw = ops.decay_powers([1.0 - 2.0 ** (-4 - 6 * j / hh) for j in range(hh)])
                x, out = torch.randn((1, 2 * hh * (d + v)), device="cuda") * 0.1, torch.empty((1, hh * v), device="cuda")
                us = time_graph([lambda s=s: ops.linear_attention(x, hh, d, v, pw, s, pos, rot, table.get(rot), 0.1, None, out) for s in states], reps)
                report(f"mixer decode {name} {hh}x{d}x{v}", us, 2 * sb + 4 * hh * (2 * d + 2 * v))
                del states
            H, D, R, V, K = la["heads"], la["dim"], la["rot"], la["vdim"], la["rank"]
            caches = [bf(n + 64, K + R, std=0.5) for _ in range(48)]
            wu = [bf(H * (D + V), K, std=0.05) for _ in range(copies(H * (D + V) * K * 2))]
            x, out = torch.randn(H * (D + R) + K + R, device="cuda"), torch.empty(H * V, device="cuda")
            ws = ops.latent_attention_workspace(H, K, R, LAYERED_WINDOW, n + 64)
            lnorm = bf(K)
            us = time_graph([lambda c=c, i=i: ops.latent_attention_decode(x, H, D, R, V, K, LAYERED_WINDOW, 0.07, 1e-5, lnorm, wu[i % len(wu)], table[R], pos, c, ws,
                                                                          out) for i, c in enumerate(caches)], reps)
            report(f"mixer decode latent attention (3 launches) {H} heads, context {n}", us, n * (K + R) * 2 + H * (D + V) * K * 2)
            del caches, wu
            ms, nq = n + 64, width // 128
            nkv = nq // 4
            q, wsp, o2 = torch.randn(nq * 128, device="cuda"), ops.single_query_attention_workspace(nq, 128, ms), torch.empty(nq * 128, device="cuda")
            kv = [(torch.randn(ms * nkv * 128, device="cuda"), torch.randn(ms * nkv * 128, device="cuda")) for _ in range(24)]
            us = time_graph([lambda c=c: ops.single_query_attention(q, c[0], c[1], n, ms, nq, nkv, 128, out=o2, workspace=wsp) for c in kv], reps)
            report(f"decode attention {nq}/{nkv} heads x 128, f32 cache, context {n} (like kernel)", us, 2 * n * nkv * 128 * 4)
            del kv
        # ---- prompt
        T = n
        if want("gemm"):
            for name, rows, cols in (("stacked q k v gate", 2 * h * (dk + dv), width), ("up", ff, width), ("down", width, ff), ("output projection", width, h * dv)):
                ws = [bf(rows, cols, std=0.02) for _ in range(4)]
                x, y = bf(T, cols), torch.empty((T, rows), dtype=torch.bfloat16, device="cuda")
                us = time_graph([lambda w=w: ops.linear_batched_bf16(x, w, out=y) for w in ws], reps)
                report(f"gemm {name} {T}x{rows}x{cols} [bf16]", us, 2 * (rows * cols + T * cols + T * rows), flops=2.0 * T * rows * cols)
                del ws
                for fmt in ("i8", "w4"):
                    ws = [_weight(fmt, rows, cols) for _ in range(4)]
                    xf, yf, sc = x.float(), torch.empty((T, rows), device="cuda"), ops.linear_batched_workspace(T, cols)
                    us = time_graph([lambda w=w: ops.linear_batched(xf, w, T, cols, rows, out=yf, workspace=sc) for w in ws], reps)
                    report(f"gemm {T}x{rows}x{cols} [{fmt}] (like kernel)", us, weight_bytes(fmt, rows, cols) + 4 * T * (rows + cols), flops=2.0 * T * rows * cols)
                    del ws, xf, yf, sc
                for m in (16, 64):  # short portions: a weight stream
                    ws = [bf(rows, cols, std=0.02) for _ in range(copies(rows * cols * 2))]
                    xm, ym, sc = bf(m, cols), torch.empty((m, rows), dtype=torch.bfloat16, device="cuda"), ops.linear_batched_bf16_workspace()
                    us = time_graph([lambda w=w: ops.linear_batched_bf16(xm, w, out=ym, workspace=sc) for w in ws], reps)
                    report(f"gemm {name} {m}x{rows}x{cols} [bf16]", us, 2 * (rows * cols + m * cols + m * rows), flops=2.0 * m * rows * cols)
                    del ws
                    for fmt in ("i8", "w4"):
                        ws = [_weight(fmt, rows, cols) for _ in range(copies(rows * cols // 2))]
                        xf, yf, sc = xm.float(), torch.empty((m, rows), device="cuda"), ops.linear_batched_workspace(m, cols)
                        us = time_graph([lambda w=w: ops.linear_batched(xf, w, m, cols, rows, out=yf, workspace=sc) for w in ws], reps)
                        report(f"gemm {m}x{rows}x{cols} [{fmt}] (like kernel)", us, weight_bytes(fmt, rows, cols) + 4 * m * (rows + cols), flops=2.0 * m * rows * cols)
                        del ws, xf, yf, sc
                torch.cuda.empty_cache()
        if want("mixer prompt"):
            for name, hh, d, v, rot in (("lightning", h, dk, dv, 0), ("retention", rh, rdk, rdv, rdk)):
                xs = [bf(T, 2 * hh * (d + v), std=0.2) for _ in range(4)]
                pw = ops.decay_powers([1.0 - 2.0 ** (-4 - 6 * j / hh) for j in range(hh)])
                st, out, sc = torch.zeros(hh * d * v, device="cuda"), torch.empty((T, hh * v), device="cuda"), ops.linear_attention_scratch(T, hh, d, v)
                us = time_graph([lambda x=x: ops.linear_attention(x, hh, d, v, pw, st, 0, rot, table.get(rot), 0.1, sc, out) for x in xs], reps)
                fl = 2.0 * hh * T * (2 * d * v + 32.5 * (d + v))  # state in and out, and on average 32.5 tokens of the chunk
                report(f"mixer prompt {name} (3 launches) {T} tokens, {hh}x{d}x{v}", us, T * hh * (2 * d * 2 + v * 2 + v * 4), flops=fl)
                del xs
            H, D, R, V, K = la["heads"], la["dim"], la["rot"], la["vdim"], la["rank"]
            x, cache, ex, out = bf(T, H * (D + R) + K + R), bf(T, K + R, std=0.5), bf(T, H * (D + V), std=0.5), torch.empty((T, H * V), device="cuda")
            us = time_graph([lambda: ops.latent_attention_prefill(x, 0, H, D, R, V, K, LAYERED_WINDOW, 0.07, table[R], cache, ex, 0, out)] * 4, reps)
            report(f"mixer prompt latent attention {T} tokens, {H} heads", us, T * (H * (D + R) + K + R + H * (D + V)) * 2 + T * H * V * 4, flops=1.0 * H * T * T * (D + R + V))
        if want("rows"):
            xs = [bf(T, ff) for _ in range(4)]
            os_ = torch.empty_like(xs[0])
            us = time_graph([lambda x=x: ops.polynorm_rows_bf16(x, coef, 1e-5, out=os_) for x in xs], reps)
            report(f"rows polynorm [{T},{ff}] bf16", us, 4 * T * ff)
            us = time_graph([lambda x=x: ops.softmax_rows(x, out=os_) for x in xs], reps) if ff <= 8192 else None
            if us:
                report(f"rows softmax [{T},{ff}] bf16 (like kernel)", us, 4 * T * ff)
            del xs
        torch.cuda.empty_cache()
        # ---- whole decoders
        if want("decoder"):
            layers, hbm = 12, peak_hbm_gbs()[0]
            dec = layered_decoder(width, layers, n + 256)
            ms, pf = time_decoder(dec, n, max(16, reps))
            wb = dec.weight_bytes - (32000 + n + 256) * width * 2
            nst = sum(1 for i in range(layers) if i % 3 != 1)
            sb = sum(2 * 4 * (h * dk * dv if i % 3 == 0 else rh * rdk * rdv) for i in range(layers) if i % 3 != 1)
            cb = (layers - nst) * n * (la["rank"] + la["rot"]) * 2
            print(json.dumps({"op": f"decoder layered {width} wide, {layers} layers", "decode_ms": round(ms, 4), "decode_tokens_per_s": round(1e3 / ms, 1),
                              "launches_per_step": dec.launches_per_step, "step_frac_hbm": round((wb + sb + cb) / ms / 1e6 / hbm, 3), "prefill_ms": round(pf, 3),
                              "prefill_tokens_per_s": round(n / pf * 1e3)}), flush=True)
            dec.close()
            heads = width // 128
            for name, fmt in (("rs_i8", rt.FORMAT_RS_I8), ("w4g128", rt.FORMAT_W4G128)):
                cfg = rt.DecoderConfig(n_layers=layers, dim=width, n_heads=heads, n_kv_heads=heads // 4, head_dim=128, hidden_dim=ff, vocab_size=32000, max_seq_len=n + 256,
                                       rope_theta=1e6, norm_eps=1e-5, format=fmt)
                dec = rt.Decoder(cfg)
                dec.init_random(7, 0.02)
                ms, pf = time_decoder(dec, n, max(16, reps))
                wb = cfg.linear_elements() * (1 if fmt == rt.FORMAT_RS_I8 else 0.515625) + layers * 2 * n * (heads // 4) * 128 * 4
                print(json.dumps({"op": f"decoder uniform {width} wide, {layers} layers, {name} (closest model)", "decode_ms": round(ms, 4),
                                  "decode_tokens_per_s": round(1e3 / ms, 1), "launches_per_step": dec.launches_per_step, "step_frac_hbm": round(wb / ms / 1e6 / hbm, 3),
                                  "prefill_ms": round(pf, 3), "prefill_tokens_per_s": round(n / pf * 1e3)}), flush=True)
                dec.close()
                torch.cuda.empty_cache()


# ---- Somopel ---------------------------------------------------------------------------------------------------------------
# sizes that resemble real layers of the given width: (heads, kv heads, head size) of the attention, (heads, dim, vdim) of both recurrences
SOMOPEL_SIZES = {4096: dict(ff=14336, attention=(32, 8, 128), gated=(32, 128, 128), delta=(32, 128, 128), rank=16, delta_rank=128),
                 2048: dict(ff=8192, attention=(16, 4, 128), gated=(16, 128, 128), delta=(16, 128, 128), rank=16, delta_rank=64)}
SOMOPEL_CHUNK = 4096


def somopel_decoder(width, layers, max_seq_len, vocab=32000, compute_f32=False, chunk=SOMOPEL_CHUNK):
    """Random-weight decoder whose layers alternate between the parallel mixer and the channel delta rule."""
    from . import runtime as rt
    from .somopel import layered_config
    z = SOMOPEL_SIZES[width]
    (H, G, D), (gh, gk, gv), (dh, dk, dv) = z["attention"], z["gated"], z["delta"]

    def layer(i):
        if i % 2 == 0:
            m = {"left": {"heads": H, "kv_heads": G, "dim": D, "vdim": D, "scale": D ** -0.5, "mask": {"size": chunk}}, "left_scale": 0.9,
                 "right": {"heads": gh, "dim": gk, "vdim": gv, "tau": 12.0}, "right_scale": 1.1}
            return {"type": "parallel", "mixer": m, "mlp": {"kind": "dense", "ff": z["ff"]}}
        return {"type": "channel_delta", "mixer": {"heads": dh, "kv_heads": dh, "dim": dk, "vdim": dv, "conv": 4}, "mlp": {"kind": "dense", "ff": z["ff"]}}

    config = {"width": width, "vocab": vocab, "max_positions": max_seq_len, "norm": {"eps": 1e-5}, "embedding": {"scale": 1.0}, "logit_scale": 1.0,
              "layers": [layer(i) for i in range(layers)]}
    dec = rt.LayeredDecoder(layered_config(config, lambda name: (z["rank"] if ".right." in name else z["delta_rank"],), compute_f32=compute_f32))
    dec.init_random(7, 0.02)
    return dec


def suite_somopel(reps, cpu=None, only="", context=2048):
    """The kernels of the Somopel design beside the like kernels of the closest model (the layered decoder of suite `layered`, at equal
    sizes; for softmax attention the uniform decoder's), then whole decoders of equal width and layer count: decode at context
    2048, 2048-token prompt.  Inputs of a line together exceed L2."""
    from . import runtime as rt
    gen = torch.Generator(device="cuda").manual_seed(6)

    def bf(*shape, std=1.0):
        return (torch.randn(shape, generator=gen, device="cuda") * std).to(torch.bfloat16)

    def want(name):
        return not only or only in name

    def copies(nbytes):
        return max(2, min(48, int(300e6 // nbytes) + 1))

    n = context
    pos = torch.tensor([n, 0, 0, 0], dtype=torch.int32, device="cuda")
    for width, z in SOMOPEL_SIZES.items():
        ff, (H, G, D), (gh, gk, gv), (dh, dk, dv) = z["ff"], z["attention"], z["gated"], z["delta"]
        att = rt.MixerSpec(rt.MIXER_ATTENTION, H, D, D, kv_heads=G, score_scale=D ** -0.5, chunk=SOMOPEL_CHUNK, head_gate=1, gate_act=rt.ACT_SIGMOID, out_scale=0.9)
        gated = rt.MixerSpec(rt.MIXER_GATED_LINEAR, gh, gk, gv, q_scale=gk ** -0.5, decay_kind=rt.DECAY_LOGISTIC, decay_tau=12.0, decay_rank=z["rank"],
                             out_norm=rt.OUT_NORM_HEAD_WEIGHTED, out_scale=1.1)
        delta = rt.MixerSpec(rt.MIXER_GATED_LINEAR, dh, dk, dv, q_scale=dk ** -0.5, decay_kind=rt.DECAY_SOFTPLUS, decay_rank=z["delta_rank"], delta=1, conv=4,
                             unit_eps=1e-6, gate_rank=z["delta_rank"], gate_act=rt.ACT_SIGMOID, out_norm=rt.OUT_NORM_HEAD_WEIGHTED)
        par_rows, del_rows = (H + 2 * G) * D + H + 2 * gh * (gk + gv) + z["rank"], dh * (2 * dk + dv) + 2 * z["delta_rank"] + dh
        # ---- one row of x
        nw, nb = bf(width), bf(width)
        shapes = [("layer norm + projections of both mixers", par_rows, width, 0), ("layer norm + projections of the delta rule", del_rows, width, 0),
                  ("layer norm + gelu(gate) up", 2 * ff, width, rt.ACT_GELU_TANH), ("layer norm + logits", 32000, width, 0)]
        if want("matvec"):
            x, y = torch.randn(width, device="cuda"), torch.empty(max(32000, 2 * ff, par_rows), device="cuda")
            for name, rows, cols, act in shapes:
                ws = [bf(rows, cols, std=0.02) for _ in range(copies(rows * cols * 2))]
                us = time_graph([lambda w=w: ops.normed_linear_bf16(x, w, rt.NORM_LAYER, nw, nb, 1e-5, act, out=y) for w in ws], reps)
                report(f"matvec {name} {rows}x{cols}", us, rows * cols * 2 + 4 * cols + 4 * rows)
                us = time_graph([lambda w=w: ops.linear_bf16(x, w, norm_weight=nw, norm_offset=1.0, eps=1e-5, out=y) for w in ws], reps)
                report(f"matvec norm + projection {rows}x{cols} (like kernel)", us, rows * cols * 2 + 4 * cols + 4 * rows)
                del ws
            cols = H * D + gh * gv
            ws = [bf(width, cols, std=0.02) for _ in range(copies(width * cols * 2))]
            o, res, hw = torch.randn(cols, device="cuda"), torch.randn(width, device="cuda"), bf(gv)
            g0, g1, y1 = torch.randn(H, device="cuda"), torch.randn(gh * gv, device="cuda"), torch.empty(width, device="cuda")
            gj = torch.randn(cols, device="cuda")
            us = time_graph([lambda w=w: ops.mixer_output_linear_bf16([att, gated], o, [None, hw], [g0, g1], w, 1e-5, res, y1) for w in ws], reps)
            report(f"matvec outputs of both mixers + projection {width}x{cols}", us, width * cols * 2 + 4 * cols + 4 * width)
            us = time_graph([lambda w=w: ops.gated_linear_bf16(o, gj, w, 1e-5, head_len=gv, residual=res, out=y1) for w in ws], reps)
            report(f"matvec gate + projection {width}x{cols} (like kernel)", us, width * cols * 2 + 4 * cols + 4 * width)
            ws = [bf(width, ff, std=0.02) for _ in range(copies(width * ff * 2))]
            xf, coef = torch.randn(ff, device="cuda"), bf(4)
            us = time_graph([lambda w=w: ops.linear_bf16(xf, w, residual=res, out=y1) for w in ws], reps)
            report(f"matvec down {width}x{ff}", us, width * ff * 2 + 4 * ff + 4 * width)
            us = time_graph([lambda w=w: ops.polynorm_linear_bf16(xf, coef, 1e-5, w, residual=res, out=y1) for w in ws], reps)
            report(f"matvec polynorm + down {width}x{ff} (like kernel)", us, width * ff * 2 + 4 * ff + 4 * width)
            del ws
        # ---- mixers, one token
        aoff, kv = (0, H * D, (H + G) * D), 2 * G * D

        def offsets(m):
            q, v = (m.kv_heads or m.heads) * m.dim, m.heads * m.vdim
            return (0, q, 2 * q, 2 * q + v, 2 * q + v + 2 * m.decay_rank, 2 * q + v + m.decay_rank)

        def weights(m, count):
            return [dict(decay_up=bf(m.heads * m.dim, m.decay_rank, std=0.1), decay_bias=bf(m.heads * m.dim), decay_log=bf(m.heads) if m.delta else None,
                         conv=bf(m.heads * (2 * m.dim + m.vdim), 4, std=0.5) if m.conv else None,
                         gate_up=bf(m.heads * m.vdim, m.gate_rank, std=0.1) if m.gate_rank else None) for _ in range(count)]

        def columns(m):
            return offsets(m)[4] + (m.heads + 7) // 8 * 8

        def extra_bytes(m):
            return 2 * m.heads * (m.dim * m.decay_rank + m.vdim * m.gate_rank) + (2 + 4) * m.conv * m.heads * (2 * m.dim + m.vdim)

        if want("mixer decode"):
            caches = [bf(n + 64, kv, std=0.5) for _ in range(48)]
            x, out = torch.randn((1, (H + 2 * G) * D), device="cuda"), torch.empty((1, H * D), device="cuda")
            us = time_graph([lambda c=c: ops.grouped_attention(att, x, aoff, pos, c, out) for c in caches], reps)
            report(f"mixer decode attention {H}/{G} heads x {D}, bf16 cache, context {n}", us, n * kv * 2)
            del caches
            caches = [(torch.randn((n + 64) * G * D, device="cuda"), torch.randn((n + 64) * G * D, device="cuda")) for _ in range(24)]
            q, wsp, o2 = torch.randn(H * D, device="cuda"), ops.single_query_attention_workspace(H, D, n + 64), torch.empty(H * D, device="cuda")
            us = time_graph([lambda c=c: ops.single_query_attention(q, c[0], c[1], n, n + 64, H, G, D, out=o2, workspace=wsp) for c in caches], reps)
            report(f"mixer decode attention {H}/{G} heads x {D}, f32 cache, context {n} (like kernel)", us, 2 * n * kv * 2)
            del caches
            for name, m in (("gated linear", gated), ("delta rule", delta)):
                sb, cnt = m.heads * m.dim * m.vdim * 4, copies(m.heads * m.dim * m.vdim * 8)
                states, ws = [torch.randn(m.heads * m.dim * m.vdim, device="cuda") for _ in range(cnt)], weights(m, cnt)
                x, out = torch.randn((1, columns(m)), device="cuda") * 0.1, torch.empty((1, m.heads * m.vdim), device="cuda")
                gate = torch.empty(m.heads * m.vdim, device="cuda")
                rings = [torch.zeros(4 * m.heads * (2 * m.dim + m.vdim), device="cuda") for _ in range(cnt)]
                us = time_graph([lambda i=i: ops.gated_linear_attention(m, x, offsets(m), pos, states[i], ring=rings[i], gate=gate, out=out, **ws[i]) for i in range(cnt)],
                                reps)
                report(f"mixer decode {name} {m.heads}x{m.dim}x{m.vdim}", us, 2 * sb + extra_bytes(m) + 4 * columns(m) + 4 * m.heads * m.vdim)
            pw = ops.decay_powers([0.99] * gh)
            xl = torch.randn((1, 2 * gh * (gk + gv)), device="cuda") * 0.1
            us = time_graph([lambda s=s: ops.linear_attention(xl, gh, gk, gv, pw, s, pos, 0, None, 0.1, None, out) for s in states], reps)
            report(f"mixer decode lightning {gh}x{gk}x{gv} (like kernel)", us, 2 * sb + 4 * gh * (2 * gk + 2 * gv))
            del states, ws, rings
        # ---- prompt
        T = n
        if want("gemm"):
            for rows, cols, act in ((par_rows, width, 0), (2 * ff, width, rt.ACT_GELU_TANH), (width, ff, 0), (width, H * D + gh * gv, 0)):
                ws = [bf(rows, cols, std=0.02) for _ in range(4)]
                x, y = bf(T, cols), torch.empty((T, rows), dtype=torch.bfloat16, device="cuda")
                if act:
                    yp = torch.empty((T, rows // 2), dtype=torch.bfloat16, device="cuda")
                    us = time_graph([lambda w=w: ops.pair_linear_batched_bf16(x, w, act, out=yp) for w in ws], reps)
                    report(f"gemm gelu(gate) up {T}x{rows}x{cols}", us, 2 * (rows * cols + T * cols + T * rows // 2), flops=2.0 * T * rows * cols)
                us = time_graph([lambda w=w: ops.linear_batched_bf16(x, w, out=y) for w in ws], reps)
                report(f"gemm {T}x{rows}x{cols}" + (" (like kernel)" if act else ""), us, 2 * (rows * cols + T * cols + T * rows), flops=2.0 * T * rows * cols)
                del ws, x, y
        if want("mixer prompt"):
            caches = [bf(T, kv, std=0.5) for _ in range(4)]
            xs, out = [bf(T, (H + 2 * G) * D) for _ in range(4)], torch.empty((T, H * D), device="cuda")
            for chunk in (SOMOPEL_CHUNK, 512):
                att.chunk = chunk
                seen = min(chunk, T)
                us = time_graph([lambda i=i: ops.grouped_attention(att, xs[i], aoff, 0, caches[i], out) for i in range(4)], reps)
                report(f"mixer prompt attention (2 launches) {T} tokens, {H}/{G} heads x {D}, chunk {chunk}", us, T * (H + 2 * G) * D * 2 + T * kv * 2 + T * H * D * 4,
                       flops=2.0 * H * T * seen * D)
            att.chunk = SOMOPEL_CHUNK
            del caches, xs
            caches = [(torch.randn(T * G * D, device="cuda"), torch.randn(T * G * D, device="cuda")) for _ in range(4)]
            q = torch.randn(T * H * D, device="cuda")
            us = time_graph([lambda c=c: ops.prefill_causal_attention(q, c[0], c[1], T, T, H, G, D, out=out.view(-1)) for c in caches], reps)
            report(f"mixer prompt attention {T} tokens, {H}/{G} heads x {D}, f32 cache (like kernel)", us, T * (H + 2 * G) * D * 4 + T * H * D * 4, flops=2.0 * H * T * T * D)
            del caches
            for name, m in (("gated linear", gated), ("delta rule", delta)):
                xs, ws = [bf(T, columns(m), std=0.2) for _ in range(4)], weights(m, 4)
                st, out, sc = torch.zeros(m.heads * m.dim * m.vdim, device="cuda"), torch.empty((T, m.heads * m.vdim), device="cuda"), ops.gated_linear_scratch(m, T)
                ring = torch.zeros(4 * m.heads * (2 * m.dim + m.vdim), device="cuda")
                us = time_graph([lambda i=i: ops.gated_linear_attention(m, xs[i], offsets(m), 0, st, ring=ring, scratch=sc, out=out, **ws[i]) for i in range(4)], reps)
                fl = 2.0 * m.heads * T * (2 * m.dim * m.vdim + 32.5 * (m.dim + m.vdim) + (m.dim * m.vdim + 65 * m.dim + 32.5 * m.vdim if m.delta else 0))
                report(f"mixer prompt {name} ({3 if m.conv else 2} launches) {T} tokens, {m.heads}x{m.dim}x{m.vdim}", us, T * m.heads * (2 * m.dim * 2 + m.vdim * 2 + m.vdim * 4),
                       flops=fl)
                del xs, ws, sc
            xs, sc = [bf(T, 2 * gh * (gk + gv), std=0.2) for _ in range(4)], ops.linear_attention_scratch(T, gh, gk, gv)
            pw, st = ops.decay_powers([0.99] * gh), torch.zeros(gh * gk * gv, device="cuda")
            us = time_graph([lambda x=x: ops.linear_attention(x, gh, gk, gv, pw, st, 0, 0, None, 0.1, sc, out) for x in xs], reps)
            report(f"mixer prompt lightning (3 launches) {T} tokens, {gh}x{gk}x{gv} (like kernel)", us, T * gh * (2 * gk * 2 + gv * 2 + gv * 4),
                   flops=2.0 * gh * T * (2 * gk * gv + 32.5 * (gk + gv)))
            del xs, sc
        if want("rows"):
            xs, os_ = [torch.randn((T, width), device="cuda") for _ in range(8)], torch.empty((T, width), dtype=torch.bfloat16, device="cuda")
            us = time_graph([lambda x=x: ops.norm_rows_bf16(x, rt.NORM_LAYER, nw, nb, 1e-5, os_) for x in xs], reps)
            report(f"rows layer norm [{T},{width}] f32 -> bf16", us, 6 * T * width)
            us = time_graph([lambda x=x: ops.norm_rows_bf16(x, rt.NORM_RMS, nw, None, 1e-5, os_) for x in xs], reps)
            report(f"rows rms norm [{T},{width}] f32 -> bf16 (like kernel)", us, 6 * T * width)
            del xs
        torch.cuda.empty_cache()
        # ---- whole decoders
        if want("decoder"):
            layers, (hbm, tensor, _) = 12, peak_hbm_gbs()
            for name, make in (("somopel", somopel_decoder), ("layered", layered_decoder)):
                dec = make(width, layers, n + 256)
                ms, pf = time_decoder(dec, n, max(16, reps))
                elements = dec.cfg.weight_elements()
                line = {"op": f"decoder {name} {width} wide, {layers} layers" + (" (closest model)" if name == "layered" else ""), "decode_ms": round(ms, 4),
                        "decode_tokens_per_s": round(1e3 / ms, 1), "launches_per_step": dec.launches_per_step, "weights_gb": round(2e-9 * elements, 3),
                        "weights_frac_hbm": round(2 * elements / ms / 1e6 / hbm, 3), "prefill_ms": round(pf, 3), "prefill_tokens_per_s": round(n / pf * 1e3),
                        "prefill_weights_frac_tensor": round(2.0 * n * (elements - 32000 * width) / pf / 1e9 / tensor, 3)}
                print(json.dumps(line), flush=True)
                dec.close()
                torch.cuda.empty_cache()


def run_decode_batch(a):
    """--batch sequences in lockstep on a Mistral-7B-shaped decoder of --layers layers, each at context --rows: the whole
    step per layer (batched linears + attention over --batch caches), small enough for a profiler capture."""
    import numpy as np

    from . import runtime as rt
    ctx, B, steps = a.rows, a.batch, max(2, a.reps)
    cfg = rt.DecoderConfig(n_layers=a.layers, dim=4096, n_heads=32, n_kv_heads=8, head_dim=128, hidden_dim=14336, vocab_size=32000,
                           rope_theta=1.0e6, norm_eps=1.0e-5, max_seq_len=ctx + steps + 24,
                           format=rt.FORMAT_RS_I8 if a.fmt == "i8" else rt.FORMAT_W4G128, kv_bf16=a.kv_bf16)
    dec = rt.Decoder(cfg)
    dec.init_random(3, 0.02, False)
    dec.prefill(np.random.default_rng(3).integers(0, cfg.vocab_size, ctx))
    bd = rt.BatchDecoder(dec, B)
    for slot in range(B):
        bd.adopt(slot)
    bd.generate_greedy(3)
    torch.cuda.synchronize()
    if a.profile:
        torch.cuda.profiler.start()
        bd.enqueue_steps(1)
        torch.cuda.synchronize()
        torch.cuda.profiler.stop()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    bd.enqueue_steps(steps)
    e1.record()
    torch.cuda.synchronize()
    ms = e0.elapsed_time(e1) / steps
    kv_bytes = a.layers * B * 2 * (ctx + 3 + steps / 2) * 1024 * (2 if a.kv_bf16 else 4)
    print(json.dumps({"op": "decode_batch", "fmt": a.fmt, "layers": a.layers, "batch": B, "context": ctx, "kv_bf16": a.kv_bf16,
                      "ms_per_step": ms, "launches_per_step": bd.launches_per_step, "kv_bytes_per_step": kv_bytes}))
    bd.close()
    dec.close()


def run_prefill(a):
    """Batched prefill of a --rows-token prompt on the Mistral-7B-shaped decoder (--layers layers; 32 = the whole model):
    wall time of the call (host clock around a synchronised call, best of three warm calls)."""
    import time

    import numpy as np

    from . import runtime as rt
    n = a.rows
    cfg = rt.DecoderConfig(n_layers=a.layers, dim=4096, n_heads=32, n_kv_heads=8, head_dim=128, hidden_dim=14336, vocab_size=32000,
                           rope_theta=1.0e6, norm_eps=1.0e-5, max_seq_len=n + 64,
                           format=rt.FORMAT_RS_I8 if a.fmt == "i8" else rt.FORMAT_W4G128, kv_bf16=a.kv_bf16)
    dec = rt.Decoder(cfg)
    dec.init_random(3, 0.02, False)
    prompt = np.random.default_rng(3).integers(0, cfg.vocab_size, n)
    dec.prefill(prompt)  # allocates the scratch
    best = None
    for _ in range(3):
        torch.cuda.synchronize()
        t0 = time.perf_counter()
        dec.prefill(prompt)
        torch.cuda.synchronize()
        dt = time.perf_counter() - t0
        best = dt if best is None else min(best, dt)
    if a.profile:
        torch.cuda.profiler.start()
        dec.prefill(prompt)
        torch.cuda.synchronize()
        torch.cuda.profiler.stop()
    print(json.dumps({"op": "prefill", "fmt": a.fmt, "layers": a.layers, "prompt_len": n, "kv_bf16": a.kv_bf16, "seconds": best,
                      "tokens_per_s": n / best}))
    dec.close()


def run_one(a):
    if a.op == "decode_batch":
        return run_decode_batch(a)
    if a.op == "prefill":
        return run_prefill(a)
    calls = []
    if a.op == "attention":
        n_heads, n_kv, hd = 32, 8, 128
        max_seq = ((a.rows + 63) // 64 + 4) * 64
        q = torch.randn(n_heads * hd, device="cuda")
        ws = ops.single_query_attention_workspace(n_heads, hd, max_seq)
        out = torch.empty(n_heads * hd, device="cuda")
        for _ in range(a.mats):
            kc, vc = torch.randn(max_seq * n_kv * hd, device="cuda"), torch.randn(max_seq * n_kv * hd, device="cuda")
            calls.append(lambda kc=kc, vc=vc: ops.single_query_attention(q, kc, vc, a.rows, max_seq, n_heads, n_kv, hd, out=out, workspace=ws))
        alg = 2 * a.rows * n_kv * hd * 4 + 2 * n_heads * hd * 4
    elif a.op == "linear_batched":
        m = a.batch
        xb = torch.randn((m, a.cols), device="cuda")
        outb = torch.empty((m, a.rows), device="cuda")
        scratch = ops.linear_batched_workspace(m, a.cols)
        for _ in range(a.mats):
            w = _weight(a.fmt, a.rows, a.cols)
            calls.append(lambda w=w: ops.linear_batched(xb, w, m, a.cols, a.rows, out=outb, workspace=scratch))
        alg = weight_bytes(a.fmt, a.rows, a.cols) + 4 * m * a.cols + 4 * m * a.rows
    else:
        x = torch.randn(a.cols, device="cuda")
        gamma = torch.ones(a.cols, dtype=torch.bfloat16, device="cuda")
        out = torch.empty(a.rows, device="cuda")
        res = torch.randn(a.rows, device="cuda")
        alg = weight_bytes(a.fmt, a.rows, a.cols) + 4 * a.cols + 4 * a.rows
        for _ in range(a.mats):
            w = _weight(a.fmt, a.rows, a.cols)
            if a.op == "linear":
                calls.append(lambda w=w: ops.linear(x, w, out=out))
            elif a.op == "qkv":  # RMSNorm + Q/K/V in one launch; rows = query rows + 2 x (rows / 6) KV rows (32q / 8kv heads)
                kv = a.rows // 6
                wk, wv = _weight(a.fmt, kv, a.cols), _weight(a.fmt, kv, a.cols)
                wq = _weight(a.fmt, a.rows - 2 * kv, a.cols)
                calls.append(lambda wq=wq, wk=wk, wv=wv: ops.linear_triple(x, wq, wk, wv, norm_weight=gamma, eps=1e-5))
            elif a.op == "linear_residual":
                calls.append(lambda w=w: ops.linear_residual(x, w, res, out=out))
            elif a.op == "linear_top1":
                calls.append(lambda w=w: ops.linear_top1(x, w))
            elif a.fmt == "w4p":
                pair = ops.DeviceW4PMatrix.from_gate_up(_weight("w4", a.rows, a.cols), _weight("w4", a.rows, a.cols))
                calls.append(lambda pair=pair: ops.silu_gate_up(x, pair, None, norm_weight=gamma, eps=1e-5, out=out))
            else:
                w2 = _weight(a.fmt, a.rows, a.cols)
                calls.append(lambda w=w, w2=w2: ops.silu_gate_up(x, w, w2, norm_weight=gamma, eps=1e-5, out=out))
        if a.op == "silu_gate_up":
            alg = 2 * weight_bytes(a.fmt, a.rows, a.cols) + 4 * a.cols + 2 * a.cols + 4 * a.rows
    for c in calls[:2]:
        c()
    torch.cuda.synchronize()
    graph = torch.cuda.CUDAGraph()
    with torch.cuda.graph(graph):
        for c in calls:
            c()
    for _ in range(3):
        graph.replay()
    torch.cuda.synchronize()
    if a.profile:
        torch.cuda.profiler.start()
        graph.replay()
        torch.cuda.synchronize()
        torch.cuda.profiler.stop()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    for _ in range(a.reps):
        graph.replay()
    e1.record()
    torch.cuda.synchronize()
    us = e0.elapsed_time(e1) * 1e3 / (a.reps * len(calls))
    line = {"op": a.op, "fmt": a.fmt, "rows": a.rows, "cols": a.cols, "us_per_launch": us, "algorithmic_bytes_per_launch": alg,
            "achieved_gbs": alg / us / 1e3}
    if a.op == "linear_batched":
        line["batch"] = a.batch
        line["tflops"] = 2.0 * a.batch * a.rows * a.cols / us / 1e6
    print(json.dumps(line))


if __name__ == "__main__":
    main()
