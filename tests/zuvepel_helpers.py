"""Small Zuvepel configurations with random weights for the tests, written out as checkpoint directories."""
from __future__ import annotations

import torch

from tafopel_helpers import tokens, write_checkpoint  # noqa: F401  (shared: token streams, checkpoint writer)


def attention(heads=4, kv_heads=2, dim=16, vdim=12, chunk=10, rot_dims=8, base=10000.0, scale=0.25):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if chunk:
        m["mask"] = {"size": chunk}
    if rot_dims:
        m["rot"] = {"dims": rot_dims, "base": base}
    return {"type": "attention", "mixer": m}


def delta(heads=4, kv_heads=2, dim=12, vdim=8, conv=3):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def gla(heads=3, dim=10, vdim=14, tau=4.0):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}}


def dense(ff=72):
    return {"kind": "dense", "ff": ff}


def config(layers, width=64, vocab=97, eps=2e-5, loop=None, scale=3.5, mult=0.45):
    cfg = {"architecture": "Zuvepel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": [dict(l, mlp=mlp) for l, mlp in layers]}
    if scale is not None:
        cfg["embedding"] = {"scale": scale}
    if mult is not None:
        cfg["residual_mult"] = mult
    if loop:
        cfg["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return cfg


def config_a():
    """every mixer kind, a loop of three layers run three times in the middle, layers without feed-forward, chunks shorter than a
    page and across pages, half-rotated heads, shared query/key heads in the delta rule."""
    return config([(gla(), dense()),
                   (attention(), dense(40)),
                   (delta(), None),
                   (gla(heads=2, dim=12, vdim=20, tau=16.0), dense(24)),
                   (attention(heads=3, kv_heads=1, dim=8, vdim=24, chunk=37, rot_dims=8, base=300.0, scale=0.3), None)], loop=(1, 4, 3))


def config_b():
    """no embedding scale, unit residual multiplier, the loop opens at the first layer and covers all of them, one head, a chunk of
    one token, no rotation, one tap, tau 1, odd sizes."""
    return config([(delta(heads=1, kv_heads=1, dim=10, vdim=6, conv=1), dense(23)),
                   (attention(heads=1, kv_heads=1, dim=12, vdim=20, chunk=1, rot_dims=0, scale=0.3), dense(36)),
                   (gla(heads=5, dim=7, vdim=9, tau=1.0), None),
                   (attention(heads=5, kv_heads=5, dim=9, vdim=4, chunk=0, rot_dims=2, base=50.0, scale=0.35), dense(8))],
                  width=45, vocab=61, eps=1e-6, loop=(0, 4, 2), scale=None, mult=None)


def config_c():
    """sizes of the tensor-core attention path (heads of 64, 32 and 128, several query heads per key/value head and one), chunks
    around the 64-key tile, 64 x 64, 128 x 40 and 48 x 72 states, no loop."""
    return config([(attention(heads=8, kv_heads=2, dim=64, vdim=64, chunk=65, rot_dims=32, scale=0.125), dense(96)),
                   (delta(heads=4, kv_heads=1, dim=64, vdim=64, conv=4), dense(64)),
                   (gla(heads=2, dim=48, vdim=72, tau=8.0), dense(48)),
                   (attention(heads=4, kv_heads=4, dim=32, vdim=128, chunk=64, rot_dims=32, scale=0.18), dense(80)),
                   (delta(heads=2, kv_heads=2, dim=128, vdim=40, conv=2), None)], width=128, vocab=211, mult=0.6)


def config_d():
    """attention only: nothing but pages remembers a prefix."""
    return config([(attention(heads=2, kv_heads=1, dim=8, vdim=8, chunk=50, rot_dims=4, scale=0.4), dense(40)),
                   (attention(heads=4, kv_heads=2, dim=8, vdim=16, chunk=0, rot_dims=8, scale=0.35), None)], width=40, vocab=50, loop=(1, 2, 2))


RANKS = {"a1": 5, "g1": 11}          # ranks of the low-rank maps: given by the tensors alone


def shapes(cfg, ranks=None):
    W, r = cfg["width"], dict(RANKS, **(ranks or {}))
    out = {"embed": (cfg["vocab"], W), "head": (cfg["vocab"], W), "final.norm": (W,), "final.norm.b": (W,)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        q = p + "mix."
        out.update({p + "norm1": (W,), p + "norm1.b": (W,)})
        H, d, vd = m["heads"], m["dim"], m["vdim"]
        if layer["type"] == "attention":
            G = m["kv_heads"]
            out.update({q + "q": (H * d, W), q + "q.b": (H * d,), q + "k": (G * d, W), q + "k.b": (G * d,), q + "v": (G * vd, W), q + "v.b": (G * vd,),
                        q + "g": (H, W)})
        elif layer["type"] == "channel_delta":
            G, K = m["kv_heads"], m["conv"]
            out.update({q + "q": (G * d, W), q + "q.conv": (G * d, K), q + "k": (G * d, W), q + "k.conv": (G * d, K), q + "v": (H * vd, W),
                        q + "v.conv": (H * vd, K), q + "b": (H, W), q + "A_log": (H,), q + "dt_bias": (H * d,), q + "a1": (r["a1"], W),
                        q + "a2": (H * d, r["a1"]), q + "g1": (r["g1"], W), q + "g2": (H * vd, r["g1"]), q + "norm": (vd,)})
        else:
            out.update({q + "q": (H * d, W), q + "k": (H * d, W), q + "v": (H * vd, W), q + "g": (H * vd, W), q + "a1": (r["a1"], W),
                        q + "a2": (H * d, r["a1"]), q + "a2.b": (H * d,), q + "norm": (vd,)})
        out[q + "o"] = (W, H * vd)
        mlp = layer.get("mlp")
        if mlp is not None:
            out.update({p + "norm2": (W,), p + "norm2.b": (W,), p + "mlp.gate": (mlp["ff"], W), p + "mlp.up": (mlp["ff"], W),
                        p + "mlp.down": (W, mlp["ff"])})
    return out


def random_weights(cfg, seed=0, ranks=None):
    """bf16 tensors (what a checkpoint holds).  Scales keep activations O(1); decays spread from one token to hundreds, differently
    in every key channel."""
    g = torch.Generator().manual_seed(seed)
    W = {}
    for name, shape in shapes(cfg, ranks).items():
        leaf = name.split(".")[-1]
        rnd = lambda s=1.0: torch.randn(shape, generator=g) * s
        if len(shape) == 1 and (leaf in ("norm1", "norm2", "norm")):
            w = 1.0 + rnd(0.3)
        elif name.endswith("a2.b"):
            w = 2.0 + rnd(1.5)
        elif leaf == "b" and len(shape) == 1:
            w = rnd(0.4)
        elif leaf == "A_log":
            w = torch.log(0.2 + 2.0 * torch.rand(shape, generator=g))
        elif leaf == "dt_bias":
            w = -2.5 + rnd(2.0)
        elif leaf == "conv":
            w = rnd(0.6)
        elif name == "embed":
            w = rnd(0.5)
        else:
            w = rnd(1.5 / shape[-1] ** 0.5)
        W[name] = w.to(torch.bfloat16)
    return W
