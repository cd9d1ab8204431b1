"""Plain implementation of the Pekunex decoder: float64, whole sequences, no cache, no batching, one function per mechanism.
Test infrastructure only: it shares no code with the product path and is written from the design's equations.

Weights: a dict name -> tensor (any float dtype; cast to float64 here).  Linear weights are [out, in] and applied as W x.

    embedding:  x = E[t] * s
    layer:      x <- x + mixer(rms(x) w1);  x <- x + ff(rms(x) w2)          (a layer may use another layer's tensors)
    rms:        y / sqrt(mean(y^2) + eps)
    mixers:     'attention'  grouped-query attention: biases, half-split rotation with interpolated frequencies, unit-RMS q and k after
                             it, soft-capped scores, an output gate per element
                'parallel'   attention with a learned sink beside a matrix memory (mLSTM), summed with two constants
                'mamba2'     state-space recurrence with one decay per head, shared B and C, gate before a grouped norm
    ff:         W_down (silu(W_gate h) * (W_up h))
    output:     logits = head (rms(x) w) * scale
"""
from __future__ import annotations

import math

import torch
import torch.nn.functional as F

F64 = torch.float64


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def unit_rms(y: torch.Tensor, eps: float) -> torch.Tensor:
    return y / torch.sqrt((y * y).mean(-1, keepdim=True) + eps)


def rms_norm(y: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return unit_rms(y, eps) * w.to(F64)


def embedding(W: dict, cfg: dict, tokens: list[int]) -> torch.Tensor:
    return W["embed"].to(F64)[tokens] * float((cfg.get("embedding") or {}).get("scale", 1.0))


def ramp_frequencies(dims: int, base: float, sc: dict | None) -> tuple[list[float], float]:
    """(frequency of every pair, magnitude of cos and sin): a linear ramp over the pair number between kept and divided frequencies."""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not sc:
        return f, 1.0
    pair_at = lambda turns: dims * math.log(float(sc["original"]) / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(pair_at(float(sc["fast"]))), 0)
    hi = min(math.ceil(pair_at(float(sc["slow"]))), dims - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / float(sc["factor"]) * r + fi * (1.0 - r))
    return out, 0.1 * math.log(float(sc["factor"])) + 1.0


def banded_frequencies(dims: int, base: float, sc: dict | None) -> list[float]:
    """Frequencies kept for short waves, divided for long ones, blended in between."""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not sc:
        return f
    factor, low, high, orig = (float(sc[k]) for k in ("factor", "low", "high", "original"))
    out = []
    for fi in f:
        wave = 2.0 * math.pi / fi
        if wave < orig / high:
            out.append(fi)
        elif wave > orig / low:
            out.append(fi / factor)
        else:
            s = (orig / wave - low) / (high - low)
            out.append((1.0 - s) * fi / factor + s * fi)
    return out


def rotate_halves(x: torch.Tensor, freq: list[float], magnitude: float = 1.0) -> torch.Tensor:
    """x [n, heads, d]: elements i and i + len(freq) of the token at position p turn by p * freq[i] and are scaled by the magnitude."""
    n, half = x.shape[0], len(freq)
    ang = torch.arange(n, dtype=F64)[:, None] * torch.tensor(freq, dtype=F64)[None, :]
    c, s = magnitude * torch.cos(ang)[:, None, :], magnitude * torch.sin(ang)[:, None, :]
    out = x.clone()
    u, v = x[..., :half], x[..., half:2 * half]
    out[..., :half] = u * c - v * s
    out[..., half:2 * half] = v * c + u * s
    return out


def causal_softmax(s: torch.Tensor, sink: float | None = None) -> torch.Tensor:
    """s [n, n]: weights over j <= i; with a sink the denominator also holds exp(sink)."""
    n = s.shape[0]
    s = torch.where(torch.arange(n)[:, None] >= torch.arange(n)[None, :], s, torch.full_like(s, -math.inf))
    if sink is None:
        return torch.softmax(s, -1)
    return torch.softmax(torch.cat([s, torch.full((n, 1), float(sink), dtype=F64)], 1), -1)[:, :n]


def gated_attention(W: dict, p: str, m: dict, h: torch.Tensor, eps: float) -> torch.Tensor:
    w = lambda leaf: W[p + leaf].to(F64)
    H, G, d, vd = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    n = h.shape[0]
    q = (h @ w("q").T + w("q.b")).view(n, H, d)
    k = (h @ w("k").T + w("k.b")).view(n, G, d)
    v = (h @ w("v").T + w("v.b")).view(n, G, vd)
    rot = m.get("rot")
    if rot and int(rot["dims"]):
        freq, mag = ramp_frequencies(int(rot["dims"]), float(rot["base"]), rot.get("scaling"))
        q, k = rotate_halves(q, freq, mag), rotate_halves(k, freq, mag)
    q, k = unit_rms(q, eps), unit_rms(k, eps)
    cap = m.get("softcap")
    o = []
    for hh in range(H):
        s = (q[:, hh] @ k[:, hh // (H // G)].T) * float(m["scale"])
        if cap:
            s = float(cap) * torch.tanh(s / float(cap))
        o.append(causal_softmax(s) @ v[:, hh // (H // G)])
    return (torch.cat(o, -1) * torch.sigmoid(h @ w("g").T)) @ w("o").T


def sink_attention(W: dict, p: str, m: dict, h: torch.Tensor) -> torch.Tensor:
    w = lambda leaf: W[p + leaf].to(F64)
    H, G, d, vd = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    n = h.shape[0]
    q, k, v = (h @ w("q").T).view(n, H, d), (h @ w("k").T).view(n, G, d), (h @ w("v").T).view(n, G, vd)
    rot = m.get("rot")
    if rot and int(rot["dims"]):
        freq = banded_frequencies(int(rot["dims"]), float(rot["base"]), rot.get("scaling"))
        q, k = rotate_halves(q, freq), rotate_halves(k, freq)
    o = []
    for hh in range(H):
        s = (q[:, hh] @ k[:, hh // (H // G)].T) * float(m["scale"])
        o.append(causal_softmax(s, float(w("sink")[hh])) @ v[:, hh // (H // G)])
    return torch.cat(o, -1) @ w("o").T


def memory_parts(q, k, v, i, f):
    """One head's matrix memory, token by token.  q, k [n, d], v [n, vd], log input gate i [n], log forget gate f [n] -> (read-out before its
    division [n, vd], normaliser n . q [n], running maximum [n])."""
    n, d, vd = q.shape[0], q.shape[1], v.shape[1]
    S, z, m = torch.zeros(d, vd, dtype=F64), torch.zeros(d, dtype=F64), 0.0
    num, nq, top = torch.empty(n, vd, dtype=F64), torch.empty(n, dtype=F64), torch.empty(n, dtype=F64)
    for t in range(n):
        new = max(float(f[t]) + m, float(i[t]))
        keep, write = math.exp(float(f[t]) + m - new), math.exp(float(i[t]) - new)
        S = keep * S + write * torch.outer(k[t], v[t])
        z = keep * z + write * k[t]
        m = new
        num[t], nq[t], top[t] = S.T @ q[t], z @ q[t], m
    return num, nq, top


def memory_cell(q, k, v, i, f):
    """-> the read-out [n, vd]: divided by the larger of |n . q| and exp(-m), plus 1e-6."""
    num, nq, top = memory_parts(q, k, v, i, f)
    return num / (torch.maximum(nq.abs(), torch.exp(-top)) + 1e-6)[:, None]


def matrix_memory(W: dict, p: str, m: dict, h: torch.Tensor, eps: float) -> torch.Tensor:
    w = lambda leaf: W[p + leaf].to(F64)
    H, d, vd, cap = int(m["heads"]), int(m["dim"]), int(m["vdim"]), float(m["gate_cap"])
    n = h.shape[0]
    q = (h @ w("q").T).view(n, H, d) * d ** -0.5
    k, v = (h @ w("k").T).view(n, H, d), (h @ w("v").T).view(n, H, vd)
    i = cap * torch.tanh((h @ w("i").T + w("i.b")) / cap)
    f = F.logsigmoid(cap * torch.tanh((h @ w("f").T + w("f.b")) / cap))
    o = torch.stack([memory_cell(q[:, a], k[:, a], v[:, a], i[:, a], f[:, a]) for a in range(H)], 1)
    o = unit_rms(o, eps).reshape(n, H * vd) * w("norm") * torch.sigmoid(h @ w("g").T)
    return o @ w("o").T


def side_by_side(W: dict, p: str, m: dict, h: torch.Tensor, eps: float) -> torch.Tensor:
    return float(m["left_scale"]) * sink_attention(W, p + "left.", m["left"], h) + \
        float(m["right_scale"]) * matrix_memory(W, p + "right.", m["right"], h, eps)


def causal_conv(x: torch.Tensor, w: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    """x [n, C], w [C, taps]: y[t, c] = b[c] + sum_j w[c, taps - 1 - j] x[t - j, c], zeros before the start."""
    n, taps = x.shape[0], w.shape[1]
    y = b[None, :].expand_as(x).clone()
    for j in range(min(taps, n)):
        y[j:] += x[:n - j] * w[:, taps - 1 - j]
    return y


def state_space(x, B, C, dt, A_log):
    """One head, token by token: S <- exp(-exp(A_log) dt) S + dt B x^T, y = S^T C.  x [n, vd], B, C [n, N], dt [n] -> [n, vd]."""
    S = torch.zeros(B.shape[1], x.shape[1], dtype=F64)
    out = torch.empty_like(x)
    for t in range(x.shape[0]):
        S = math.exp(-math.exp(float(A_log)) * float(dt[t])) * S + float(dt[t]) * torch.outer(B[t], x[t])
        out[t] = S.T @ C[t]
    return out


def mamba2(W: dict, p: str, m: dict, h: torch.Tensor, eps: float) -> torch.Tensor:
    w = lambda leaf: W[p + leaf].to(F64)
    H, vd, N, G, ng = int(m["heads"]), int(m["vdim"]), int(m["state"]), int(m["groups"]), int(m.get("norm_groups") or 1)
    n, inner = h.shape[0], H * vd
    z, xbc, dt = torch.split(h @ w("in").T, [inner, inner + 2 * G * N, H], 1)
    xbc = silu(causal_conv(xbc, w("conv"), w("conv.b")))
    x, B, C = xbc[:, :inner].reshape(n, H, vd), xbc[:, inner:inner + G * N].reshape(n, G, N), xbc[:, inner + G * N:].reshape(n, G, N)
    dt = F.softplus(dt + w("dt_bias"))
    y = torch.empty(n, H, vd, dtype=F64)
    for a in range(H):
        g = a // (H // G)
        y[:, a] = state_space(x[:, a], B[:, g], C[:, g], dt[:, a], w("A_log")[a]) + w("D")[a] * x[:, a]
    y = y.reshape(n, inner) * silu(z)
    y = unit_rms(y.view(n, ng, inner // ng), eps).reshape(n, inner) * w("norm")
    return y @ w("o").T


def dense_ff(W: dict, p: str, h: torch.Tensor) -> torch.Tensor:
    w = lambda leaf: W[p + leaf].to(F64)
    return (silu(h @ w("gate").T) * (h @ w("up").T)) @ w("down").T


def forward(cfg: dict, W: dict, tokens: list[int], taps: list | None = None) -> torch.Tensor:
    """-> logits [n, vocab] (float64).  ``taps`` collects the residual stream after every layer."""
    eps = float(cfg["norm"]["eps"])
    x = embedding(W, cfg, tokens)
    for i, layer in enumerate(cfg["layers"]):
        owner = i
        while cfg["layers"][owner].get("weights_of") is not None:
            owner = int(cfg["layers"][owner]["weights_of"])
        p = f"l{owner}."
        h = rms_norm(x, W[p + "norm1"], eps)
        mixer = {"attention": gated_attention, "parallel": side_by_side, "mamba2": mamba2}[layer["type"]]
        x = x + mixer(W, p + "mix.", layer["mixer"], h, eps)
        if layer.get("mlp") is not None:
            x = x + dense_ff(W, p + "mlp.", rms_norm(x, W[p + "norm2"], eps))
        if taps is not None:
            taps.append(x.clone())
    return rms_norm(x, W["final.norm"], eps) @ W["head"].to(F64).T * float(cfg.get("logit_scale", 1.0))
