"""Small Pekunex configurations with random weights for the tests, written out as checkpoint directories."""
from __future__ import annotations

import torch

from tafopel_helpers import tokens, write_checkpoint  # noqa: F401  (shared: token streams, checkpoint writer)

RAMP = {"factor": 5.0, "original": 40, "fast": 6.0, "slow": 0.5}             # short enough for kept, blended and divided pairs within few dimensions
BANDS = {"factor": 3.0, "original": 64, "low": 0.5, "high": 6.0}


def attention(heads=4, kv_heads=2, dim=20, vdim=12, rot_dims=12, base=900.0, scaling=RAMP, scale=0.3, softcap=4.0):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if softcap is not None:
        m["softcap"] = softcap
    if rot_dims:
        m["rot"] = dict({"dims": rot_dims, "base": base}, **({"scaling": scaling} if scaling else {}))
    return {"type": "attention", "mixer": m}


def left(heads=3, kv_heads=1, dim=12, vdim=10, rot_dims=8, base=700.0, scaling=BANDS, scale=0.35):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if rot_dims:
        m["rot"] = dict({"dims": rot_dims, "base": base}, **({"scaling": scaling} if scaling else {}))
    return m


def right(heads=2, dim=14, vdim=18, gate_cap=7.0):
    return {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": gate_cap}


def parallel(l=None, r=None, left_scale=0.7, right_scale=1.3):
    return {"type": "parallel", "mixer": {"left": l or left(), "right": r or right(), "left_scale": left_scale, "right_scale": right_scale}}


def mamba2(heads=6, vdim=10, state=12, groups=3, conv=4, norm_groups=2):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}}


def dense(ff=72):
    return {"kind": "dense", "ff": ff}


def config(layers, width=64, vocab=97, eps=2e-5, scale=2.5, logit_scale=1.5):
    """layers: (entry, mlp) or the number of an earlier layer whose weights are used."""
    out = []
    for l in layers:
        out.append(dict(out[l], weights_of=l) if isinstance(l, int) else dict(l[0], mlp=l[1]))
    cfg = {"architecture": "Pekunex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": out}
    if scale is not None:
        cfg["embedding"] = {"scale": scale}
    if logit_scale is not None:
        cfg["logit_scale"] = logit_scale
    return cfg


def config_a():
    """every mixer kind, each of them run again with borrowed weights, partly rotated heads, layers without feed-forward."""
    return config([(mamba2(), dense()), (parallel(), dense(40)), (attention(), None), 0, 1, (mamba2(heads=2, vdim=24, state=9, groups=1, conv=2, norm_groups=1), None), 2])


def config_b():
    """one head everywhere, one tap, one group per head, no rotation, no scaling, no cap, no embedding or logit factor, odd sizes."""
    return config([(parallel(left(heads=1, kv_heads=1, dim=9, vdim=7, rot_dims=0), right(heads=1, dim=5, vdim=3, gate_cap=2.0), 1.0, 1.0), dense(23)),
                   (attention(heads=1, kv_heads=1, dim=11, vdim=13, rot_dims=10, scaling=None, softcap=None, scale=0.3), dense(36)),
                   (mamba2(heads=5, vdim=7, state=3, groups=5, conv=1, norm_groups=5), None),
                   (parallel(left(heads=5, kv_heads=5, dim=6, vdim=4, rot_dims=6, scaling=None), right(heads=3, dim=7, vdim=9, gate_cap=15.0)), None)],
                  width=45, vocab=61, eps=1e-6, scale=None, logit_scale=None)


def config_c():
    """sizes of the tensor-core attention, exact and zero-padded (128, 64, 32, 72, 40), and of wider states (64 x 64, 128 x 40, 96 x 80)."""
    return config([(attention(heads=8, kv_heads=2, dim=64, vdim=64, rot_dims=32, base=10000.0, scale=0.125, softcap=20.0), dense(96)),
                   (mamba2(heads=4, vdim=64, state=128, groups=2, conv=4, norm_groups=4), dense(64)),
                   (parallel(left(heads=4, kv_heads=2, dim=72, vdim=40, rot_dims=72, scale=0.12), right(heads=2, dim=64, vdim=64)), dense(48)),
                   (attention(heads=6, kv_heads=6, dim=32, vdim=128, rot_dims=32, scale=0.2, softcap=8.0), dense(80)),
                   (parallel(left(heads=2, kv_heads=1, dim=128, vdim=32, rot_dims=64, scale=0.1), right(heads=2, dim=96, vdim=80, gate_cap=4.0)), None),
                   1], width=128, vocab=211)


def config_d():
    """attention only: nothing but pages remembers a prefix."""
    return config([(attention(heads=2, kv_heads=1, dim=8, vdim=8, rot_dims=4, scale=0.5), dense(40)),
                   (attention(heads=4, kv_heads=4, dim=16, vdim=24, rot_dims=16, scale=0.35, softcap=2.0), None), 0], width=40, vocab=50)


def shapes(cfg):
    W = cfg["width"]
    out = {"embed": (cfg["vocab"], W), "head": (cfg["vocab"], W), "final.norm": (W,)}
    for i, layer in enumerate(cfg["layers"]):
        if layer.get("weights_of") is not None:
            continue
        p, m = f"l{i}.", layer["mixer"]
        q = p + "mix."
        out[p + "norm1"] = (W,)
        if layer["type"] == "attention":
            H, G, d, vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            out.update({q + "q": (H * d, W), q + "q.b": (H * d,), q + "k": (G * d, W), q + "k.b": (G * d,), q + "v": (G * vd, W), q + "v.b": (G * vd,),
                        q + "g": (H * vd, W), q + "o": (W, H * vd)})
        elif layer["type"] == "parallel":
            l, r = m["left"], m["right"]
            H, G, d, vd = l["heads"], l["kv_heads"], l["dim"], l["vdim"]
            out.update({q + "left.q": (H * d, W), q + "left.k": (G * d, W), q + "left.v": (G * vd, W), q + "left.sink": (H,), q + "left.o": (W, H * vd)})
            H, d, vd = r["heads"], r["dim"], r["vdim"]
            out.update({q + "right.q": (H * d, W), q + "right.k": (H * d, W), q + "right.v": (H * vd, W), q + "right.g": (H * vd, W),
                        q + "right.o": (W, H * vd), q + "right.norm": (H * vd,), q + "right.i": (H, W), q + "right.i.b": (H,), q + "right.f": (H, W),
                        q + "right.f.b": (H,)})
        else:
            H, vd, N, G, K = m["heads"], m["vdim"], m["state"], m["groups"], m["conv"]
            C = H * vd + 2 * G * N
            out.update({q + "in": (H * vd + C + H, W), q + "conv": (C, K), q + "conv.b": (C,), q + "dt_bias": (H,), q + "A_log": (H,), q + "D": (H,),
                        q + "norm": (H * vd,), q + "o": (W, H * vd)})
        if layer.get("mlp") is not None:
            ff = layer["mlp"]["ff"]
            out.update({p + "norm2": (W,), p + "mlp.gate": (ff, W), p + "mlp.up": (ff, W), p + "mlp.down": (W, ff)})
    return out


def random_weights(cfg, seed=0):
    """bf16 tensors (what a checkpoint holds).  Scales keep activations O(1); decays and gates spread from one token to hundreds, differently
    in every head."""
    g = torch.Generator().manual_seed(seed)
    W = {}
    for name, shape in shapes(cfg).items():
        leaf = name.split(".")[-1]
        rnd = lambda s=1.0: torch.randn(shape, generator=g) * s
        if leaf in ("norm1", "norm2", "norm", "D"):
            w = 1.0 + rnd(0.3)
        elif name.endswith("i.b"):
            w = rnd(2.0)
        elif name.endswith("f.b"):
            w = 3.0 + rnd(2.0)
        elif leaf == "b":
            w = rnd(0.4)
        elif leaf == "sink":
            w = rnd(1.5)
        elif leaf == "A_log":
            w = torch.log(0.2 + 2.0 * torch.rand(shape, generator=g))
        elif leaf == "dt_bias":
            w = -2.0 + rnd(1.5)
        elif leaf == "conv":
            w = rnd(0.6)
        elif name == "embed":
            w = rnd(0.5)
        else:
            w = rnd(1.5 / shape[-1] ** 0.5)
        W[name] = w.to(torch.bfloat16)
    return W
