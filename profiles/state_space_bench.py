"""Prefill / decode throughput of the Pekunex decoder (pre-norm layers; attention with unit-RMS queries and keys, soft cap and element gate;
sink attention beside a matrix memory; state-space recurrence) beside Zuvepel, Tafopel, Tipetar and Qwen3 at equal width, number of layer
runs and feed-forward size, plus a per-kernel roofline table of its kernels and their counterparts (``python bench.py --state-space``).

Same rules as hybrid_bench.py, whose engine set-up, throughput loop and timing helper it uses: random weights, synthetic token
ids, device time between CUDA events after warm-up, a 256 MB write between the timed launches of the per-kernel table.
"""
from __future__ import annotations

import json
import os
import sys
import time

import channel_bench as cb  # noqa: F401  (registers the Zuvepel configuration)
import hybrid_bench as hb
import window_bench as wb  # noqa: F401  (registers the Tipetar configuration)

ROOT = hb.ROOT
VOCAB = hb.VOCAB

SIZES = {
    # name: (width, heads, kv_heads, memory heads, state-space heads, groups)  -- attention heads and memory 128 wide, state-space heads of
    # 64 x 128 (inner = 2 x width); eight layers, one of them on borrowed weights
    "w1024": (1024, 16, 4, 8, 32, 2),
    "w2048": (2048, 16, 4, 16, 64, 8),
}


def pekunex_config(size: str):
    from nanovllm.models.pekunex import PekunexConfig
    width, H, G, mh, sh, gr = SIZES[size]
    ramp = {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}
    bands = {"factor": 8.0, "original": 8192, "low": 1.0, "high": 4.0}
    att = {"type": "attention", "mixer": {"heads": H, "kv_heads": G, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "softcap": 50.0,
                                          "rot": {"dims": 64, "base": 5e5, "scaling": ramp}}}
    par = {"type": "parallel", "mixer": {"left": {"heads": H // 2, "kv_heads": G // 2, "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                                                  "rot": {"dims": 128, "base": 5e5, "scaling": bands}},
                                         "right": {"heads": mh, "dim": 128, "vdim": 128, "gate_cap": 15.0}, "left_scale": 0.7, "right_scale": 0.7}}
    ssm = {"type": "mamba2", "mixer": {"heads": sh, "vdim": 64, "state": 128, "groups": gr, "conv": 4, "norm_groups": gr}}
    mlp = {"kind": "dense", "ff": 3 * width}
    layers = [dict(l, mlp=mlp) for l in (ssm, par, att, ssm, par, att, ssm)]
    return PekunexConfig({"architecture": "Pekunex", "vocab": VOCAB, "width": width, "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0}, "logit_scale": 0.5,
                          "layers": layers + [dict(layers[4], weights_of=4)]})


hb.EXTRA_KINDS["pekunex"] = pekunex_config


def kernel_table(size: str, peaks: dict):
    import torch
    from nanovllm import mixops
    from nanovllm.layers.rotary_embedding import build_banded_cos_sin
    width, H, G, mh, sh, gr = SIZES[size]
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

    # ---- attention: cap + element gate, learned sink, a padded head size; the plain form beside them ----
    for label, S, q, k in (("prefill 4x2048", 4, 2048, 2048), ("decode 64x4096", 64, 1, 4096)):
        nblk = S * (k // bs)
        n, spn = S * q, spans(S, q, k)
        bt = torch.arange(nblk, dtype=torch.int32, device=dev).view(S, -1)
        pairs = S * (sum(i + 1 for i in range(q)) if q > 1 else k)
        for name, hd, kw in (("cap + element gate", d, dict(softcap=50.0, gate=rn(n, H * d))), ("learned sink", d, dict(sinks=torch.zeros(H, device=dev))),
                             ("cap + element gate, heads of 96", 96, dict(softcap=50.0, gate=rn(n, H * 96))), ("plain (tipetar form)", d, {})):
            cache, qkv = rn(nblk * bs, G * 2 * hd), rn(n, H * hd)
            nbytes = S * k * G * 2 * hd * 2 + n * H * hd * (6 if "gate" in kw else 4)
            add(f"window_attention {name} {label}", lambda: mixops.window_attention(qkv, cache, bt, bs, spn, H, G, hd, hd, 0.088, **kw), nbytes,
                pairs * H * 4 * hd, "tensor")
    # ---- rotation, norm and cache store; the form without norms beside it ----
    n = 8192
    table = build_banded_cos_sin(64, 8192, 5e5, None, dev)
    qkv, cache = rn(n, (H + 2 * G) * d), torch.zeros(n, G * 2 * d, dtype=bf, device=dev)
    sl, pos = torch.arange(n, dtype=torch.int32, device=dev), torch.arange(n, dtype=torch.int64, device=dev)
    store = lambda unit: mixops.headnorm_rope_store(qkv, 0, H * d, (H + G) * d, H, G, d, d, None, None, False, table, pos, sl, cache, 1e-6,
                                                    layout=mixops.ROT_HALVES, unit_after=unit)
    add("rope_store, unit norm after the rotation 8192 rows", lambda: store(True), n * ((2 * H + 4 * G) * d) * 2, 0)
    add("rope_store, no norms (zuvepel form) 8192 rows", lambda: store(False), n * ((2 * H + 4 * G) * d) * 2, 0)
    # ---- matrix states: prompt steps and a decode step; linear attention with channel decays beside them ----
    for label, S, q in (("prefill 4x2048", 4, 2048), ("prefill 64x1024", 64, 1024), ("decode 64", 64, 1)):
        n = S * q
        spn, slots = spans(S, q, q if q > 1 else 100), torch.arange(S, dtype=torch.int32, device=dev)
        C = sh * 64 + 2 * gr * d
        x, step, st = rn(n, C), rn(n, sh), torch.zeros(S, sh, 64, d, device=dev)
        rate, bias = -torch.rand(sh, device=dev), torch.zeros(sh, device=dev)
        add(f"linear_state, state space {label}", lambda: mixops.linear_state(x, sh * 64 + gr * d, sh * 64, 0, st, slots, spn, sh, gr, d, 64, step=step, rate=rate,
            bias=bias), n * (C * 2 + sh * 2 + sh * 64 * 4) + 2 * st.numel() * 4, n * sh * 64 * d * 5, "fma")
        if q > 1:
            add(f"linear_state, state space, fp32-pipe form {label}", lambda: mixops.linear_state(x, sh * 64 + gr * d, sh * 64, 0, st, slots, spn, sh, gr, d, 64,
                step=step, rate=rate, bias=bias, fma=True), n * (C * 2 + sh * 2 + sh * 64 * 4) + 2 * st.numel() * 4, n * sh * 64 * d * 5, "fma")
        y, z, wn, D = torch.randn(n, sh, 64, device=dev), rn(n, sh * 64), rn(sh * 64), torch.ones(sh, device=dev)
        if q != 1024:
            add(f"skip_gate_groupnorm {label}", lambda: mixops.skip_gate_groupnorm(y, x[:, :sh * 64], D, z, wn, gr, 1e-6), n * sh * 64 * 10, 0)
            wc, bc, cs = rn(C, 4), rn(C), torch.zeros(S, 3, C, device=dev)
            add(f"causal_conv {label}", lambda: mixops.causal_conv(x, wc, bc, cs, slots, spn), n * C * 4, 0)
        del x, y, z
        xg, ld, wr = rn(n, 3 * mh * d), -torch.rand(n, mh, device=dev), torch.rand(n, mh, device=dev)
        sm = torch.zeros(S, mh, d + 1, d, device=dev)
        add(f"linear_state, matrix memory {label}", lambda: mixops.linear_state(xg, 0, mh * d, 2 * mh * d, sm, slots, spn, mh, mh, d, d, d ** -0.5, log_decay=ld,
            write=wr, ones=True), n * (3 * mh * d * 2 + mh * (d + 1) * 4 + mh * 8) + 2 * sm.numel() * 4, n * mh * d * (d + 1) * 5, "fma")
        if q > 1:
            add(f"linear_state, matrix memory, fp32-pipe form {label}", lambda: mixops.linear_state(xg, 0, mh * d, 2 * mh * d, sm, slots, spn, mh, mh, d, d,
                d ** -0.5, log_decay=ld, write=wr, ones=True, fma=True), n * (3 * mh * d * 2 + mh * (d + 1) * 4 + mh * 8) + 2 * sm.numel() * 4,
                n * mh * d * (d + 1) * 5, "fma")
        zz, db, sg = torch.randn(n, mh * d, device=dev), torch.zeros(mh * d, device=dev), torch.zeros(S, mh, d, d, device=dev)
        add(f"channel_state, linear attention (zuvepel form) {label}", lambda: mixops.channel_state(xg, 0, mh * d, 2 * mh * d, None, zz, rate[:mh], db, -1.0, sg,
            slots, spn, mh, mh, d, d, d ** -0.5), n * (3 * mh * d * 2 + mh * d * 8) + 2 * sg.numel() * 4, n * mh * d * d * 5, "fma")
        if q == 1024:
            continue
        pre, b2, ms = torch.randn(n, 2 * mh, device=dev), torch.zeros(2 * mh, device=dev), torch.zeros(S, mh, device=dev)
        add(f"mlstm_gates {label}", lambda: mixops.mlstm_gates(pre, b2, 15.0, ms, slots, spn, mh), n * mh * 20, 0)
        o, gz, wn, fl = torch.randn(n, mh, d + 1, device=dev), rn(n, mh * d), rn(mh * d), torch.rand(n, mh, device=dev)
        add(f"head_rmsnorm_gate, divided read-out {label}", lambda: mixops.head_rmsnorm_gate(o, wn, gz, 1e-6, bf, silu=False, floor=fl), n * mh * d * 8, 0)
        o2 = torch.randn(n, mh, d, device=dev)
        add(f"head_rmsnorm_gate (zuvepel form) {label}", lambda: mixops.head_rmsnorm_gate(o2, wn[:d], gz, 1e-6, bf, silu=False), n * mh * d * 8, 0)
    # ---- row-wise ops, 8192 rows ----
    n = 8192
    x, y = torch.randn(n, width, device=dev), rn(n, width)
    w, w2, b, b2 = rn(width), rn(width), rn(width), rn(width)
    add("add_rmsnorm 8192 rows", lambda: mixops.add_rmsnorm(x, w, 1e-6, y=y), n * width * (8 + 2 + 2), 0)
    add("add_layernorm2, two norms (zuvepel form) 8192 rows", lambda: mixops.add_layernorm2(x, 1e-6, y=y, mult=0.5, norm1=(w, b), norm2=(w2, b2)), n * width * (8 + 2 + 4), 0)
    gu = rn(n, 6 * width)
    add("ff_act silu * up 8192 rows", lambda: mixops.ff_act(gu, mixops.FF_SILU_MUL), n * 3 * width * 6, 0)
    add("ff_act gelu * up (zuvepel form) 8192 rows", lambda: mixops.ff_act(gu, mixops.FF_GELU_TANH_MUL), n * 3 * width * 6, 0)
    return rows


def main(argv=None):
    import argparse
    ap = argparse.ArgumentParser()
    ap.add_argument("--sizes", default="w1024,w2048")
    ap.add_argument("--batch", type=int, default=64)
    ap.add_argument("--prompt", type=int, default=1024)
    ap.add_argument("--new-tokens", type=int, default=48)
    ap.add_argument("--kinds", default="pekunex,zuvepel,tafopel,tipetar,qwen3")
    ap.add_argument("--no-kernels", action="store_true")
    a = ap.parse_args(argv)
    peaks = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "source": "fallback"}
    pk = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.exists(pk):
        peaks = dict(json.load(open(pk)), source="measured")
    out = {"bench": "state-space", "dtype": "bf16", "data": "synthetic token ids, random weights", "peaks": {k: peaks[k] for k in ("hbm_gbs", "bf16_tflops", "source")},
           "workload": {"batch": a.batch, "prompt": a.prompt, "new_tokens": a.new_tokens}, "sizes": {}}
    for size in a.sizes.split(","):
        t0 = time.time()
        entry = {"dims": dict(zip(("width", "heads", "kv_heads", "memory_heads", "state_space_heads", "groups"), SIZES[size]))}
        for kind in filter(None, a.kinds.split(",")):
            entry[kind] = hb.throughput(kind, size, a.batch, a.prompt, a.new_tokens)
        if not a.no_kernels:
            entry["kernels"] = kernel_table(size, peaks)
        entry["seconds"] = round(time.time() - t0, 1)
        out["sizes"][size] = entry
        print(json.dumps({size: entry}), file=sys.stderr, flush=True)
    print(json.dumps(out))


if __name__ == "__main__":
    main()
