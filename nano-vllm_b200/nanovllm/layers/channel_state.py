"""Matrix-state mixers whose decay is one number per head and KEY CHANNEL: the delta rule with channel decays and gated linear
attention.  Per head a state S [dim, vdim] (fp32, from zero), read out with the query after the token's own write.

Channel delta (``ChannelDeltaMixer``):
    q = silu(conv(W_q h)), k = silu(conv(W_k h))  [kv_heads, dim]        v = silu(conv(W_v h))  [heads, vdim]      (depthwise causal, no bias)
    q <- q / sqrt(|q|^2 + 1e-6) * dim^-1/2,  k <- k / sqrt(|k|^2 + 1e-6)                (head h reads q/k head h // (heads / kv_heads))
    beta = sigmoid(W_b h)  per head          g = exp(-exp(A_log_h) softplus(W_a2 (W_a1 h) + dt_bias))  [heads, dim]
    S <- diag(g) S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
    out = W_o (o / rms(o) * w_norm * sigmoid(W_g2 (W_g1 h)))

Gated linear attention (``GatedLinearAttention``):
    q = W_q h * dim^-1/2, k = W_k h  [heads, dim],  v = W_v h  [heads, vdim]
    alpha = sigmoid(W_a2 (W_a1 h) + b_a2)^(1 / tau)  [heads, dim]
    S <- diag(alpha) S + k v^T;  o = S^T q
    out = W_o (o / rms(o) * w_norm * silu(W_g h))

(norm per head over vdim, weight shared by the heads.)  Both decays are exp(rate_h softplus(sign (z + bias))): rate = -exp(A_log), sign 1,
and rate = -1 / tau, sign -1.  Everything narrow rides in the wide input projection: the low-rank maps' first factors and the
write strengths; the second factors are small GEMMs, the decays' one with an fp32 result.  The ranks are not in the configuration:
the first factors' shapes give them (``set_ranks``).  Decays, strengths, unit norms and the state never leave fp32
(``mixops.channel_state``).  ``w_o`` may be a view into an output projection shared with another branch, whose operand ``mix`` fills.
"""
from __future__ import annotations

import torch
import torch.nn.functional as F

from .. import mixops


def _pad8(n: int) -> int:
    return -(-n // 8) * 8


class _ChannelStateMixer:
    """What the two share: state slots, the merged input projection with parts of known and of declared sizes, the decay maps."""
    decay_sign = 1.0

    def __init__(self, width: int, m: dict, eps: float, dtype, device, w_o=None, ranks: dict | None = None):
        self.width, self.eps, self.dtype, self.device = width, eps, dtype, device
        self.heads = int(m["heads"])
        self.kv_heads = int(m.get("kv_heads", self.heads))
        self.dim, self.vdim = int(m["dim"]), int(m["vdim"])
        if self.heads % self.kv_heads:
            raise ValueError("heads must be a multiple of kv_heads")
        if self.dim > 256:
            raise ValueError(f"dim {self.dim}: the matrix-state kernel holds at most 256 state rows per column")
        self.qk_cols, self.v_cols = self.kv_heads * self.dim, self.heads * self.vdim
        self.out_cols = self.v_cols
        self.w_o = w_o if w_o is not None else torch.empty(width, self.out_cols, dtype=dtype, device=device)
        assert self.w_o.shape == (width, self.out_cols)
        self.norm_w = torch.empty(self.vdim, dtype=dtype, device=device)
        self.rate = torch.zeros(self.heads, dtype=torch.float32, device=device)
        self.decay_bias = torch.zeros(self.heads * self.dim, dtype=torch.float32, device=device)
        self.state: list = []          # per instance [slots, heads, vdim, dim] fp32
        self._mm_f32_out = dtype != torch.float32
        self.ranks: dict = {}
        self.set_ranks(dict({leaf: self.dim for leaf, _ in self.low_rank()}, **(ranks or {})))

    # ---- the parts of the input projection ---------------------------------------------------------------------------------
    def parts(self) -> list[tuple[str, int]]:
        """(leaf, rows) of the parts of known size, in order."""
        raise NotImplementedError

    def low_rank(self) -> list[tuple[str, int]]:
        """(leaf of the first factor, output columns of the second factor); the second factor's leaf ends in 2 instead of 1."""
        raise NotImplementedError

    @staticmethod
    def operand_cols(m: dict) -> int:
        return int(m["heads"]) * int(m["vdim"])

    def set_ranks(self, ranks: dict) -> None:
        """(Re)allocate the projections for these ranks (leaf of a first factor -> its rows)."""
        new = dict(self.ranks, **{k: int(v) for k, v in ranks.items()})
        if new == self.ranks:
            return
        self.ranks = new
        at, self.at = 0, {}
        for leaf, rows in self.parts():
            self.at[leaf] = (at, rows)
            at += rows
        for leaf, _ in self.low_rank():                   # each starts on a 16-byte column and fills whole 16-byte pieces
            at = _pad8(at)
            self.at[leaf] = (at, new[leaf])
            at = _pad8(at + new[leaf])
        self.in_cols = _pad8(at)
        self.w_in = torch.zeros(self.in_cols, self.width, dtype=self.dtype, device=self.device)
        self.second = {leaf[:-1] + "2": torch.zeros(cols, _pad8(new[leaf]), dtype=self.dtype, device=self.device) for leaf, cols in self.low_rank()}

    def _cols(self, proj: torch.Tensor, leaf: str) -> torch.Tensor:
        a, rows = self.at[leaf]
        return proj[:, a:a + rows]

    def _second(self, proj: torch.Tensor, leaf: str, f32: bool) -> torch.Tensor:
        """The low-rank map's result: its first factor's (zero-padded) columns of the projection times the second factor."""
        w = self.second[leaf[:-1] + "2"]
        a = self.at[leaf][0]
        t = proj[:, a:a + w.shape[1]]
        if f32 and self._mm_f32_out:
            try:
                return torch.mm(t, w.t(), out_dtype=torch.float32)
            except (RuntimeError, TypeError):
                self._mm_f32_out = False
        y = F.linear(t, w)
        return y.float() if f32 else y

    def load(self, leaf: str, w: torch.Tensor) -> bool:
        if leaf in self.at:
            a, rows = self.at[leaf]
            self.w_in[a:a + rows].copy_(w)
        elif leaf in self.second:
            self.second[leaf][:, :w.shape[1]].copy_(w)
        elif leaf == "norm":
            self.norm_w.copy_(w)
        elif leaf == "o":
            self.w_o.copy_(w)
        else:
            return False
        return True

    def weight_shapes(self, width: int) -> dict:
        out = {leaf: (rows, width) for leaf, (_, rows) in self.at.items()}
        out.update({leaf[:-1] + "2": (cols, self.ranks[leaf]) for leaf, cols in self.low_rank()})
        return dict(out, norm=(self.vdim,), o=(width, self.out_cols))

    # ---- state -------------------------------------------------------------------------------------------------------------
    def cache_row_elems(self) -> int:
        return 0

    def state_slot_bytes(self) -> int:
        return 4 * self.heads * self.vdim * self.dim

    def bind(self, num_blocks: int, block_size: int, num_slots: int, copies: int = 1) -> None:
        self.state = [torch.zeros(num_slots, self.heads, self.vdim, self.dim, dtype=torch.float32, device=self.device) for _ in range(copies)]

    def unbind(self) -> None:
        self.state = []

    def mix(self, h, positions, ctx, spans, inst: int = 0, out: torch.Tensor | None = None) -> torch.Tensor:
        raise NotImplementedError

    def forward(self, h: torch.Tensor, positions, ctx, spans: mixops.StepSpans, inst: int = 0) -> torch.Tensor:
        return F.linear(self.mix(h, positions, ctx, spans, inst), self.w_o)


class ChannelDeltaMixer(_ChannelStateMixer):
    kind = "channel_delta"

    def __init__(self, width: int, m: dict, eps: float, dtype, device, w_o=None, ranks: dict | None = None):
        self.taps = int(m["conv"])
        super().__init__(width, m, eps, dtype, device, w_o, ranks)
        self.conv_cols = 2 * self.qk_cols + self.v_cols                   # [q | k | v]: one convolution over concatenated channels
        self.conv_w = torch.empty(self.conv_cols, self.taps, dtype=dtype, device=device)
        self.conv_state: list = []     # per instance [slots, taps - 1, conv_cols] fp32

    def parts(self):
        return [("q", self.qk_cols), ("k", self.qk_cols), ("v", self.v_cols), ("b", self.heads)]

    def low_rank(self):
        return [("a1", self.heads * self.dim), ("g1", self.v_cols)]

    def load(self, leaf: str, w: torch.Tensor) -> bool:
        if leaf in ("q.conv", "k.conv", "v.conv"):
            a, rows = self.at[leaf[0]]
            self.conv_w[a:a + rows].copy_(w)
        elif leaf == "A_log":
            self.rate.copy_(-torch.exp(w.float()))
        elif leaf == "dt_bias":
            self.decay_bias.copy_(w.float().reshape(-1))
        else:
            return super().load(leaf, w)
        return True

    def weight_shapes(self, width: int) -> dict:
        K = self.taps
        return dict(super().weight_shapes(width), **{"q.conv": (self.qk_cols, K), "k.conv": (self.qk_cols, K), "v.conv": (self.v_cols, K)},
                    A_log=(self.heads,), dt_bias=(self.heads * self.dim,))

    def state_slot_bytes(self) -> int:
        return super().state_slot_bytes() + 4 * max(self.taps - 1, 1) * self.conv_cols

    def bind(self, num_blocks: int, block_size: int, num_slots: int, copies: int = 1) -> None:
        super().bind(num_blocks, block_size, num_slots, copies)
        self.conv_state = [torch.zeros(num_slots, max(self.taps - 1, 1), self.conv_cols, dtype=torch.float32, device=self.device) for _ in range(copies)]

    def unbind(self) -> None:
        super().unbind()
        self.conv_state = []

    def mix(self, h: torch.Tensor, positions, ctx, spans: mixops.StepSpans, inst: int = 0, out: torch.Tensor | None = None) -> torch.Tensor:
        """-> the output projection's operand [n, heads * vdim]."""
        Q = self.qk_cols
        proj = F.linear(h, self.w_in)
        qkv = mixops.causal_conv(proj[:, :self.conv_cols], self.conv_w, None, self.conv_state[inst], ctx.state_slots, spans)
        o = mixops.channel_state(qkv, 0, Q, 2 * Q, self._cols(proj, "b"), self._second(proj, "a1", True), self.rate, self.decay_bias,
                                 self.decay_sign, self.state[inst], ctx.state_slots, spans, self.heads, self.kv_heads, self.dim, self.vdim,
                                 self.dim ** -0.5)
        return mixops.head_rmsnorm_gate(o, self.norm_w, self._second(proj, "g1", False), self.eps, self.dtype, silu=False, out=out)


class GatedLinearAttention(_ChannelStateMixer):
    kind = "gla"
    decay_sign = -1.0

    def __init__(self, width: int, m: dict, eps: float, dtype, device, w_o=None, ranks: dict | None = None):
        super().__init__(width, dict(m, kv_heads=m["heads"]), eps, dtype, device, w_o, ranks)
        self.rate.fill_(-1.0 / float(m["tau"]))

    def parts(self):
        return [("q", self.qk_cols), ("k", self.qk_cols), ("v", self.v_cols), ("g", self.v_cols)]

    def low_rank(self):
        return [("a1", self.heads * self.dim)]

    def load(self, leaf: str, w: torch.Tensor) -> bool:
        if leaf == "a2.b":
            self.decay_bias.copy_(w.float().reshape(-1))
            return True
        return super().load(leaf, w)

    def weight_shapes(self, width: int) -> dict:
        return dict(super().weight_shapes(width), **{"a2.b": (self.heads * self.dim,)})

    def mix(self, h: torch.Tensor, positions, ctx, spans: mixops.StepSpans, inst: int = 0, out: torch.Tensor | None = None) -> torch.Tensor:
        """-> the output projection's operand [n, heads * vdim]."""
        Q = self.qk_cols
        proj = F.linear(h, self.w_in)
        o = mixops.channel_state(proj, 0, Q, 2 * Q, None, self._second(proj, "a1", True), self.rate, self.decay_bias, self.decay_sign,
                                 self.state[inst], ctx.state_slots, spans, self.heads, self.kv_heads, self.dim, self.vdim, self.dim ** -0.5)
        return mixops.head_rmsnorm_gate(o, self.norm_w, self._cols(proj, "g"), self.eps, self.dtype, silu=True, out=out)
