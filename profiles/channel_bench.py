"""Prefill / decode throughput of the Zuvepel decoder (parallel layers over two biased norms; chunked attention with a sink and head
gates, delta rule with channel decays, gated linear attention; repeated layers) beside Musavik, Tafopel, Tipetar and Qwen3 at equal
width, number of layer runs and feed-forward size, plus a per-kernel roofline table of its kernels and their counterparts
(``python bench.py --channel``).

Same rules as hybrid_bench.py, whose engine set-up, throughput loop and timing helper it uses: random weights, synthetic token
ids, device time between CUDA events after warm-up, a 256 MB write between the timed launches of the per-kernel table.
"""
from __future__ import annotations

import json
import os
import sys
import time

import hybrid_bench as hb
import recurrent_bench as rb  # noqa: F401  (registers the Musavik configuration)
import window_bench as wb  # noqa: F401  (registers the Tipetar configuration)

ROOT = hb.ROOT
VOCAB = hb.VOCAB

SIZES = {
    # name: (width, heads, kv_heads, chunk, state heads, delta q/k heads)  -- head size 128; six layers of which layers 3..4 run twice:
    # eight layer runs, as many as the eight layers of the models beside it
    "w1024": (1024, 16, 4, 1024, 8, 4),
    "w2048": (2048, 16, 4, 2048, 16, 4),
}


def zuvepel_config(size: str):
    from nanovllm.models.zuvepel import ZuvepelConfig
    width, H, G, chunk, sh, dg = SIZES[size]
    att = {"type": "attention", "mixer": {"heads": H, "kv_heads": G, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "mask": {"size": chunk},
                                          "rot": {"dims": 64, "base": 5e5}}}
    delta = {"type": "channel_delta", "mixer": {"heads": sh, "kv_heads": dg, "dim": 128, "vdim": 128, "conv": 4}}
    gla = {"type": "gla", "mixer": {"heads": sh, "dim": 128, "vdim": 128, "tau": 16.0}}
    mlp = {"kind": "dense", "ff": 3 * width}
    return ZuvepelConfig({"architecture": "Zuvepel", "vocab": VOCAB, "width": width, "norm": {"eps": 1e-6}, "embedding": {"scale": width ** 0.5},
                          "residual_mult": 0.5, "layers": [dict(l, mlp=mlp) for l in (att, delta, gla, att, delta, gla)],
                          "loop": {"start": 3, "stop": 5, "times": 2}})


hb.EXTRA_KINDS["zuvepel"] = zuvepel_config


def kernel_table(size: str, peaks: dict):
    import torch
    from nanovllm import mixops
    from nanovllm.layers.rotary_embedding import build_banded_cos_sin
    width, H, G, chunk, sh, dg = SIZES[size]
    d, bs, dev, bf = 128, 256, "cuda", torch.bfloat16
    hbm, tc = peaks["hbm_gbs"] * 1e9, peaks["bf16_tflops"] * 1e12
    fma = 148 * 128 * 2 * 1.9e9
    flush = torch.zeros(64 << 20, dtype=torch.float32, device=dev)
    rows = []

    def add(name, fn, nbytes, flops, pipe="hbm"):
        t = hb.timed(fn, flush)
        peak = tc if pipe == "tensor" else fma
        roof = max(nbytes / hbm, flops / peak if flops else 0.0)
        rows.append(dict(kernel=name, us=round(t * 1e6, 1), gbs=round(nbytes / t / 1e9, 1), tflops=round(flops / t / 1e12, 2),
                         bound="hbm" if nbytes / hbm >= (flops / peak if flops else 0) else pipe, of_roofline=round(roof / t, 3)))

    g = torch.Generator(device=dev).manual_seed(0)
    rn = lambda *s, dt=bf: torch.randn(*s, generator=g, device=dev, dtype=torch.float32).to(dt)

    def spans(S, q, k):
        if q > 1:
            cu = torch.arange(0, S + 1, dtype=torch.int32, device=dev)
            return mixops.StepSpans(S, q, cu * q, cu * k, None)
        return mixops.StepSpans(S, 1, None, None, torch.full((S,), k, dtype=torch.int32, device=dev))

    # ---- attention: chunk + sink + head gate; the plain windowed form beside it ----
    sinks = torch.zeros(H, device=dev)
    for label, S, q, k in (("prefill 4x2048", 4, 2048, 2048), ("decode 64x4096", 64, 1, 4096)):
        nblk = S * (k // bs)
        cache = rn(nblk * bs, G * 2 * d)
        bt = torch.arange(nblk, dtype=torch.int32, device=dev).view(S, -1)
        n = S * q
        qkv, gate, spn = rn(n, H * d), rn(n, H), spans(S, q, k)
        for chunked in (True, False):
            vis = (lambda i: i % chunk + 1) if chunked else (lambda i: min(i + 1, chunk))
            pairs = S * (sum(vis(i) for i in range(q)) if q > 1 else vis(k - 1))
            keys_read = S * (k if q > 1 else vis(k - 1))
            nbytes = keys_read * G * 2 * d * 2 + n * H * d * 4
            kw = dict(chunk=chunk, sinks=sinks, gate=gate) if chunked else dict(window=chunk)
            name = "window_attention chunk + sink + gate" if chunked else "window_attention window (tipetar form)"
            add(f"{name} {label}", lambda: mixops.window_attention(qkv, cache, bt, bs, spn, H, G, d, d, 0.088, **kw), nbytes, pairs * H * 4 * d, "tensor")
    # ---- rotation and cache store; Musavik's normed form beside it ----
    n = 8192
    table = build_banded_cos_sin(64, 8192, 5e5, None, dev)
    qkv, cache = rn(n, (H + 2 * G) * d), torch.zeros(n, G * 2 * d, dtype=bf, device=dev)
    sl, pos, w1 = torch.arange(n, dtype=torch.int32, device=dev), torch.arange(n, dtype=torch.int64, device=dev), rn(d)
    store = lambda norm, lay: mixops.headnorm_rope_store(qkv, 0, H * d, (H + G) * d, H, G, d, d, w1 if norm else None, w1 if norm else None, norm, table,
                                                         pos, sl, cache, 1e-6, layout=lay)
    add("rope_store, half-split pairs, no norms 8192 rows", lambda: store(False, mixops.ROT_HALVES), n * ((2 * H + 4 * G) * d) * 2, 0)
    add("headnorm_rope_store (musavik form) 8192 rows", lambda: store(True, mixops.ROT_PAIRS), n * ((2 * H + 4 * G) * d) * 2, 0)
    # ---- matrix states: a prompt step of 4 x 2048 tokens and a decode step of 64 rows; Musavik's scalar-decay delta rule beside them ----
    for label, S, q in (("prefill 4x2048", 4, 2048), ("prefill 64x1024", 64, 1024), ("decode 64", 64, 1)):
        n = S * q
        spn, slots = spans(S, q, q if q > 1 else 100), torch.arange(S, dtype=torch.int32, device=dev)
        rt, hb0 = -torch.rand(sh, device=dev), torch.zeros(sh, device=dev)
        db, state = torch.zeros(sh * d, device=dev), torch.zeros(S, sh, d, d, device=dev)
        z, st_bytes, flops = torch.randn(n, sh * d, device=dev), 2 * S * sh * d * d * 4, n * sh * d * d * 6
        x, wr, ba = rn(n, (2 * dg + sh) * d), rn(n, sh), torch.randn(n, 2 * sh, device=dev)
        add(f"channel_state, delta rule {label}", lambda: mixops.channel_state(x, 0, dg * d, 2 * dg * d, wr, z, rt, db, 1.0, state, slots, spn, sh, dg, d, d, d ** -0.5),
            n * ((2 * dg + sh) * d * 2 + sh * d * 8) + st_bytes, flops, "fma")
        add(f"gated_delta (musavik form) {label}", lambda: mixops.gated_delta(x, 0, dg * d, 2 * dg * d, ba, rt, hb0, state, slots, spn, sh, dg, d, d, d ** -0.5),
            n * ((2 * dg + sh) * d * 2 + sh * d * 4) + st_bytes, flops, "fma")
        xg = rn(n, 3 * sh * d)
        add(f"channel_state, linear attention {label}", lambda: mixops.channel_state(xg, 0, sh * d, 2 * sh * d, None, z, rt, db, -1.0, state, slots, spn, sh, sh, d, d,
            d ** -0.5), n * (3 * sh * d * 2 + sh * d * 8) + st_bytes, n * sh * d * d * 5, "fma")
        if q == 1024:
            continue
        o, gz, wn = torch.randn(n, sh, d, device=dev), rn(n, sh * d), rn(d)
        add(f"head_rmsnorm_gate {label}", lambda: mixops.head_rmsnorm_gate(o, wn, gz, 1e-6, bf, silu=False), n * sh * d * 8, 0)
        C = (2 * dg + sh) * d
        wc, cs = rn(C, 4), torch.zeros(S, 3, C, device=dev)
        add(f"causal_conv {label}", lambda: mixops.causal_conv(x, wc, None, cs, slots, spn), n * C * 4, 0)
    # ---- row-wise ops, 8192 rows ----
    n = 8192
    x, y = torch.randn(n, width, device=dev), rn(n, width)
    w, w2, b, b2 = rn(width), rn(width), rn(width), rn(width)
    x0 = torch.randn(n, width, device=dev)
    add("add_layernorm2, two norms 8192 rows", lambda: mixops.add_layernorm2(x, 1e-6, y=y, mult=0.5, norm1=(w, b), norm2=(w2, b2)), n * width * (8 + 2 + 4), 0)
    add("add_layernorm2, two norms + embedding output 8192 rows", lambda: mixops.add_layernorm2(x, 1e-6, y=y, mult=0.5, add=x0, norm1=(w, b), norm2=(w2, b2)),
        n * width * (8 + 2 + 4 + 4), 0)
    add("add_layernorm (tafopel form) 8192 rows", lambda: mixops.add_layernorm(x, w, 1e-6, a=y), n * width * (8 + 2 + 2), 0)
    add("add_normed_norm (musavik form) 8192 rows", lambda: mixops.add_normed_norm(x, y, w, 1e-6, 1.0, next_weight=w2, next_offset=1.0), n * width * (8 + 2 + 2), 0)
    ff, oc = 3 * width, H * d
    gu, both = rn(n, 2 * ff), torch.empty(n, oc + ff, dtype=bf, device=dev)
    add("ff_act gelu * up into a column slice 8192 rows", lambda: mixops.ff_act(gu, mixops.FF_GELU_TANH_MUL, out=both[:, oc:]), n * ff * 6, 0)
    add("ff_act gelu * up (tafopel form) 8192 rows", lambda: mixops.ff_act(gu, mixops.FF_GELU_TANH_MUL), n * ff * 6, 0)
    return rows


def main(argv=None):
    import argparse
    ap = argparse.ArgumentParser()
    ap.add_argument("--sizes", default="w1024,w2048")
    ap.add_argument("--batch", type=int, default=64)
    ap.add_argument("--prompt", type=int, default=1024)
    ap.add_argument("--new-tokens", type=int, default=48)
    ap.add_argument("--no-kernels", action="store_true")
    ap.add_argument("--no-models", action="store_true")
    a = ap.parse_args(argv)
    peaks = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "source": "fallback"}
    pk = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.exists(pk):
        peaks = dict(json.load(open(pk)), source="measured")
    out = {"bench": "channel", "dtype": "bf16", "data": "synthetic token ids, random weights", "peaks": {k: peaks[k] for k in ("hbm_gbs", "bf16_tflops", "source")},
           "workload": {"batch": a.batch, "prompt": a.prompt, "new_tokens": a.new_tokens}, "sizes": {}}
    for size in a.sizes.split(","):
        t0 = time.time()
        entry = {"dims": dict(zip(("width", "heads", "kv_heads", "chunk", "state_heads", "delta_qk_heads"), SIZES[size]))}
        for kind in () if a.no_models else ("zuvepel", "musavik", "tafopel", "tipetar", "qwen3"):
            entry[kind] = hb.throughput(kind, size, a.batch, a.prompt, a.new_tokens)
        if not a.no_kernels:
            entry["kernels"] = kernel_table(size, peaks)
        entry["seconds"] = round(time.time() - t0, 1)
        out["sizes"][size] = entry
        print(json.dumps({size: entry}), file=sys.stderr, flush=True)
    print(json.dumps(out))


if __name__ == "__main__":
    main()
