"""Plain implementation of the Zuvepel decoder: float64, whole sequences, no cache, no batching, one function per mechanism.
Test infrastructure only: it shares no code with the product path and is written from the design's equations.

Weights: a dict name -> tensor (any float dtype; cast to float64 here).  Linear weights are [out, in] and applied as W x.

    embedding:    x0 = E[t] * s
    layer order:  layers [start, stop) run `times` times in a row with the same weights; every pass but the first opens with x <- x + x0
    layer:        x <- x + m (mixer(ln1(x)) + ff(ln2(x)))                                (both read the same x)
    ln:           (y - mean(y)) / sqrt(mean((y - mean)^2) + eps) * w + b
    mixers:       'attention'     grouped-query attention inside chunks, half-split rotation, a zero-score sink, one gate per head
                  'channel_delta' delta rule with a decay per head and key channel
                  'gla'           gated linear attention with a decay per head and key channel
    ff:           W_down (gelu_tanh(W_gate h) * (W_up h))
    output:       logits = head ln(x)
"""
from __future__ import annotations

import math

import torch
import torch.nn.functional as F

F64 = torch.float64


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def unit_rms(y: torch.Tensor, eps: float) -> torch.Tensor:
    return y / torch.sqrt((y * y).mean(-1, keepdim=True) + eps)


def layer_norm(y: torch.Tensor, w: torch.Tensor, b: torch.Tensor, eps: float) -> torch.Tensor:
    c = y - y.mean(-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(-1, keepdim=True) + eps) * w.to(F64) + b.to(F64)


def embedding(W: dict, cfg: dict, tokens: list[int]) -> torch.Tensor:
    return W["embed"].to(F64)[tokens] * float((cfg.get("embedding") or {}).get("scale", 1.0))


def causal_conv(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """x [n, C], w [C, taps]: y[t, c] = sum_j w[c, taps - 1 - j] x[t - j, c], zeros before the start."""
    n, taps = x.shape[0], w.shape[1]
    y = torch.zeros_like(x)
    for j in range(min(taps, n)):
        y[j:] += x[:n - j] * w[:, taps - 1 - j]
    return y


def rotate_halves(x: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """x [n, heads, d]: elements i and i + dims / 2 (i < dims / 2) of the token at position p turn by p * base^(-2i / dims)."""
    n, half = x.shape[0], dims // 2
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=F64)
    ang = torch.arange(n, dtype=F64)[:, None] * f[None, :]
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    out = x.clone()
    u, v = x[..., :half], x[..., half:dims]
    out[..., :half] = u * c - v * s
    out[..., half:dims] = v * c + u * s
    return out


def same_chunk(n: int, chunk: int) -> torch.Tensor:
    """[n, n] bool: query i sees key j when j <= i and both lie in one chunk (chunk 0: every earlier key)."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    return (j <= i) & (torch.ones(n, n, dtype=torch.bool) if chunk <= 0 else i // chunk == j // chunk)


def sink_softmax(s: torch.Tensor, see: torch.Tensor) -> torch.Tensor:
    """exp(s_j) / (1 + sum_j exp(s_j)) over the visible j."""
    s = torch.where(see, s, torch.full_like(s, -math.inf))
    top = s.max(-1, keepdim=True).values.clamp(min=0.0)
    e = torch.exp(s - top)
    return e / (torch.exp(-top) + e.sum(-1, keepdim=True))


def attention(W: dict, p: str, m: dict, h: torch.Tensor) -> torch.Tensor:
    w = lambda leaf: W[p + leaf].to(F64)
    H, G, d, vd = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    n = h.shape[0]
    q = (h @ w("q").T + w("q.b")).view(n, H, d)
    k = (h @ w("k").T + w("k.b")).view(n, G, d)
    v = (h @ w("v").T + w("v.b")).view(n, G, vd)
    rot = m.get("rot")
    if rot:
        q = rotate_halves(q, int(rot["dims"]), float(rot["base"]))
        k = rotate_halves(k, int(rot["dims"]), float(rot["base"]))
    see = same_chunk(n, int((m.get("mask") or {}).get("size") or 0))
    gate = torch.sigmoid(h @ w("g").T)                                              # [n, H]
    o = []
    for hh in range(H):
        g = hh // (H // G)
        P = sink_softmax((q[:, hh] @ k[:, g].T) * float(m["scale"]), see)
        o.append((P @ v[:, g]) * gate[:, hh:hh + 1])
    return torch.cat(o, -1) @ w("o").T


def channel_delta(W: dict, p: str, m: dict, h: torch.Tensor, eps: float) -> torch.Tensor:
    """Per head a matrix state S [dim, vdim]:  S <- diag(g) S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q."""
    w = lambda leaf: W[p + leaf].to(F64)
    H, G, d, vd = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    n = h.shape[0]
    q = silu(causal_conv(h @ w("q").T, w("q.conv"))).view(n, G, d)
    k = silu(causal_conv(h @ w("k").T, w("k.conv"))).view(n, G, d)
    v = silu(causal_conv(h @ w("v").T, w("v.conv"))).view(n, H, vd)
    q = q / torch.sqrt((q * q).sum(-1, keepdim=True) + 1e-6) * d ** -0.5
    k = k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
    beta = torch.sigmoid(h @ w("b").T)                                               # [n, H]
    z = ((h @ w("a1").T) @ w("a2").T + w("dt_bias")).view(n, H, d)
    decay = torch.exp(-torch.exp(w("A_log"))[None, :, None] * F.softplus(z))         # [n, H, d]
    out = torch.empty(n, H, vd, dtype=F64)
    for hh in range(H):
        g = hh // (H // G)
        S = torch.zeros(d, vd, dtype=F64)
        for t in range(n):
            S = decay[t, hh][:, None] * S
            u = beta[t, hh] * (v[t, hh] - S.T @ k[t, g])
            S = S + torch.outer(k[t, g], u)
            out[t, hh] = S.T @ q[t, g]
    out = unit_rms(out, eps) * w("norm")
    out = out.reshape(n, H * vd) * torch.sigmoid((h @ w("g1").T) @ w("g2").T)
    return out @ w("o").T


def gla(W: dict, p: str, m: dict, h: torch.Tensor, eps: float) -> torch.Tensor:
    """Per head a matrix state S [dim, vdim]:  S <- diag(alpha) S + k v^T;  o = S^T q;  alpha = sigmoid(z)^(1 / tau)."""
    w = lambda leaf: W[p + leaf].to(F64)
    H, d, vd, tau = int(m["heads"]), int(m["dim"]), int(m["vdim"]), float(m["tau"])
    n = h.shape[0]
    q = (h @ w("q").T).view(n, H, d) * d ** -0.5
    k = (h @ w("k").T).view(n, H, d)
    v = (h @ w("v").T).view(n, H, vd)
    alpha = torch.sigmoid((h @ w("a1").T) @ w("a2").T + w("a2.b")).view(n, H, d) ** (1.0 / tau)
    out = torch.empty(n, H, vd, dtype=F64)
    for hh in range(H):
        S = torch.zeros(d, vd, dtype=F64)
        for t in range(n):
            S = alpha[t, hh][:, None] * S + torch.outer(k[t, hh], v[t, hh])
            out[t, hh] = S.T @ q[t, hh]
    out = unit_rms(out, eps) * w("norm")
    return (out.reshape(n, H * vd) * silu(h @ w("g").T)) @ w("o").T


def dense_ff(W: dict, p: str, h: torch.Tensor) -> torch.Tensor:
    w = lambda leaf: W[p + leaf].to(F64)
    return (gelu_tanh(h @ w("gate").T) * (h @ w("up").T)) @ w("down").T


def layer_runs(cfg: dict) -> list[tuple[int, bool]]:
    """(layer index, whether the embedding output is added right before it) in execution order."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    runs = [(i, False) for i in range(a)]
    for k in range(times):
        runs += [(i, i == a and k > 0) for i in range(a, b)]
    return runs + [(i, False) for i in range(b, n)]


def forward(cfg: dict, W: dict, tokens: list[int], taps: list | None = None) -> torch.Tensor:
    """-> logits [n, vocab] (float64).  ``taps`` collects the residual stream after every layer run."""
    eps, mult = float(cfg["norm"]["eps"]), float(cfg.get("residual_mult", 1.0))
    x0 = embedding(W, cfg, tokens)
    x = x0
    for i, reopened in layer_runs(cfg):
        if reopened:
            x = x + x0
        layer, p = cfg["layers"][i], f"l{i}."
        h = layer_norm(x, W[p + "norm1"], W[p + "norm1.b"], eps)
        if layer["type"] == "attention":
            y = attention(W, p + "mix.", layer["mixer"], h)
        elif layer["type"] == "channel_delta":
            y = channel_delta(W, p + "mix.", layer["mixer"], h, eps)
        elif layer["type"] == "gla":
            y = gla(W, p + "mix.", layer["mixer"], h, eps)
        else:
            raise ValueError(layer["type"])
        if layer.get("mlp") is not None:
            y = y + dense_ff(W, p + "mlp.", layer_norm(x, W[p + "norm2"], W[p + "norm2.b"], eps))
        x = x + mult * y
        if taps is not None:
            taps.append(x.clone())
    return layer_norm(x, W["final.norm"], W["final.norm.b"], eps) @ W["head"].to(F64).T
