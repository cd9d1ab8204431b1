"""Matrix-state mixers with one decay and one write weight per token and HEAD, ``S <- g S + w k v^T``, ``o = S^T q`` (S fp32, from zero):
a state-space recurrence (Mamba-2) and the matrix memory of xLSTM.  Both run the same kernel (``mixops.linear_state``).

State space (``StateSpaceMixer``), inner = heads * vdim:
    [z : inner | x : inner | B : groups * state | C : groups * state | dt : heads] = W_in h
    (x, B, C) <- silu(conv(x, B, C) + b)                        (depthwise causal over the concatenated channels)
    w = softplus(dt + dt_bias),  g = exp(-exp(A_log) w),  k = B, v = x, q = C        (head h reads group h // (heads / groups))
    y = o + D_h x;   out = W_o (groupnorm(y * silu(z)) * w_norm)                      (each of norm_groups equal parts by its own root mean square)

Matrix memory (``MatrixMemoryMixer``):
    q = W_q h * dim^-1/2,  k = W_k h  [heads, dim],   v = W_v h  [heads, vdim]
    i = cap tanh((W_i h + b_i) / cap),   f = logsigmoid(cap tanh((W_f h + b_f) / cap))             (logarithms of the gates, one per head)
    m' = max(f + m, i),  g = exp(f + m - m'),  w = exp(i - m'),  m <- m'                            (m from 0)
    n <- g n + w k;   o <- S^T q / (max(|n . q|, exp(-m)) + 1e-6)
    out = W_o (o / rms(o) * w_norm * sigmoid(W_g h))                                                (rms per head, weight per head and element)
  n is one more column of S whose value is always 1, so the same kernel carries and reads it.  The gates' pre-activations come from a small
  GEMM with an fp32 result, the running maximum and what follows from it from one scan in front of the states (``mixops.mlstm_gates``).

Per sequence and instance a state slot holds S, and the last taps - 1 convolution inputs or m.  Decays, write weights, the running
maximum and the states never leave fp32.
"""
from __future__ import annotations

import torch
import torch.nn.functional as F

from .. import mixops

MAX_DIM = 256          # state rows per column the matrix-state kernels hold


class StateSpaceMixer:
    kind = "mamba2"

    def __init__(self, width: int, m: dict, eps: float, dtype, device, max_position: int | None = None):
        self.width, self.eps, self.dtype, self.device = width, eps, dtype, device
        self.heads, self.vdim, self.nstate, self.groups = int(m["heads"]), int(m["vdim"]), int(m["state"]), int(m["groups"])
        self.taps, self.norm_groups = int(m["conv"]), int(m.get("norm_groups") or 1)
        self.inner = self.heads * self.vdim
        if self.heads % self.groups or self.inner % self.norm_groups:
            raise ValueError("heads must be a multiple of groups, and heads * vdim of norm_groups")
        if self.nstate > MAX_DIM:
            raise ValueError(f"state {self.nstate}: the matrix-state kernels hold at most {MAX_DIM} state rows per column")
        self.bc = self.groups * self.nstate
        self.conv_cols = self.inner + 2 * self.bc                          # [x | B | C]
        self.dt_off = self.inner + self.conv_cols
        self.in_cols = self.dt_off + self.heads
        e = lambda *s: torch.empty(*s, dtype=dtype, device=device)
        self.w_in = torch.zeros(-(-self.in_cols // 8) * 8, width, dtype=dtype, device=device)        # whole 16-byte rows of the result
        self.conv_w, self.conv_b = e(self.conv_cols, self.taps), e(self.conv_cols)
        self.norm_w, self.w_o = e(self.inner), e(width, self.inner)
        z = lambda: torch.zeros(self.heads, dtype=torch.float32, device=device)
        self.rate, self.dt_bias, self.D = z(), z(), z()                    # -exp(A_log)
        self.conv_state: list = []     # per instance [slots, taps - 1, conv_cols] fp32
        self.state: list = []          # per instance [slots, heads, vdim, state] fp32

    def load(self, leaf: str, w: torch.Tensor) -> bool:
        named = {"conv": self.conv_w, "conv.b": self.conv_b, "norm": self.norm_w, "o": self.w_o}
        if leaf == "in":
            self.w_in[:self.in_cols].copy_(w)
        elif leaf == "A_log":
            self.rate.copy_(-torch.exp(w.float()))
        elif leaf in ("dt_bias", "D"):
            getattr(self, leaf).copy_(w.float())
        elif leaf in named:
            named[leaf].copy_(w)
        else:
            return False
        return True

    def weight_shapes(self, width: int) -> dict:
        H = self.heads
        return {"in": (self.in_cols, width), "conv": (self.conv_cols, self.taps), "conv.b": (self.conv_cols,), "dt_bias": (H,), "A_log": (H,), "D": (H,),
                "norm": (self.inner,), "o": (width, self.inner)}

    def cache_row_elems(self) -> int:
        return 0

    def state_slot_bytes(self) -> int:
        return 4 * (max(self.taps - 1, 1) * self.conv_cols + self.inner * self.nstate)

    def bind(self, num_blocks: int, block_size: int, num_slots: int, copies: int = 1) -> None:
        z = lambda *s: torch.zeros(*s, dtype=torch.float32, device=self.device)
        self.conv_state = [z(num_slots, max(self.taps - 1, 1), self.conv_cols) for _ in range(copies)]
        self.state = [z(num_slots, self.heads, self.vdim, self.nstate) for _ in range(copies)]

    def unbind(self) -> None:
        self.conv_state, self.state = [], []

    def rotations(self):
        return []

    def forward(self, h: torch.Tensor, positions, ctx, spans: mixops.StepSpans, inst: int = 0) -> torch.Tensor:
        I, Q = self.inner, self.bc
        proj = F.linear(h, self.w_in)
        xbc = mixops.causal_conv(proj[:, I:self.dt_off], self.conv_w, self.conv_b, self.conv_state[inst], ctx.state_slots, spans)
        y = mixops.linear_state(xbc, I + Q, I, 0, self.state[inst], ctx.state_slots, spans, self.heads, self.groups, self.nstate, self.vdim,
                                step=proj[:, self.dt_off:self.in_cols], rate=self.rate, bias=self.dt_bias)
        return F.linear(mixops.skip_gate_groupnorm(y, xbc[:, :I], self.D, proj[:, :I], self.norm_w, self.norm_groups, self.eps), self.w_o)


class MatrixMemoryMixer:
    """Input projection ``[W_q ; W_k ; W_v ; W_g]`` and output projection may be views into the merged weights of a block that runs this
    mixer beside another one on the same input (``ParallelMixer``)."""
    kind = "mlstm"

    def __init__(self, width: int, m: dict, eps: float, dtype, device, w_in=None, w_o=None):
        self.width, self.eps, self.dtype, self.device = width, eps, dtype, device
        self.heads, self.dim, self.vdim, self.cap = int(m["heads"]), int(m["dim"]), int(m["vdim"]), float(m["gate_cap"])
        if self.dim > MAX_DIM:
            raise ValueError(f"dim {self.dim}: the matrix-state kernels hold at most {MAX_DIM} state rows per column")
        H = self.heads
        self.qk_cols, self.v_cols = H * self.dim, H * self.vdim
        self.in_cols, self.out_cols = self.projection_cols(m)
        e = lambda *s: torch.empty(*s, dtype=dtype, device=device)
        self.w_in = w_in if w_in is not None else e(self.in_cols, width)
        self.w_o = w_o if w_o is not None else e(width, self.out_cols)
        assert self.w_in.shape == (self.in_cols, width) and self.w_o.shape == (width, self.out_cols)
        self.w_if = e(2 * H, width)                                        # [W_i ; W_f]: fp32 result
        self.b_if = torch.zeros(2 * H, dtype=torch.float32, device=device)
        self.norm_w = e(self.v_cols)
        self.state: list = []          # per instance [slots, heads, vdim + 1, dim] fp32: S and, as the last column, n
        self.m_state: list = []        # per instance [slots, heads] fp32
        self._mm_f32_out = dtype != torch.float32

    @staticmethod
    def projection_cols(m: dict) -> tuple[int, int]:
        """(rows of the wide input projection, columns of the output projection) for a mixer configuration."""
        qk, v = int(m["heads"]) * int(m["dim"]), int(m["heads"]) * int(m["vdim"])
        return 2 * qk + 2 * v, v

    def load(self, leaf: str, w: torch.Tensor) -> bool:
        Q, V, H = self.qk_cols, self.v_cols, self.heads
        spans = {"q": (0, Q), "k": (Q, 2 * Q), "v": (2 * Q, 2 * Q + V), "g": (2 * Q + V, self.in_cols)}
        if leaf in spans:
            self.w_in[spans[leaf][0]:spans[leaf][1]].copy_(w)
        elif leaf in ("i", "f"):
            self.w_if[H * (leaf == "f"):H + H * (leaf == "f")].copy_(w)
        elif leaf in ("i.b", "f.b"):
            self.b_if[H * (leaf == "f.b"):H + H * (leaf == "f.b")].copy_(w.float())
        elif leaf == "norm":
            self.norm_w.copy_(w)
        elif leaf == "o":
            self.w_o.copy_(w)
        else:
            return False
        return True

    def weight_shapes(self, width: int) -> dict:
        Q, V, H = self.qk_cols, self.v_cols, self.heads
        return {"q": (Q, width), "k": (Q, width), "v": (V, width), "g": (V, width), "i": (H, width), "i.b": (H,), "f": (H, width), "f.b": (H,),
                "norm": (V,), "o": (width, V)}

    def cache_row_elems(self) -> int:
        return 0

    def state_slot_bytes(self) -> int:
        return 4 * self.heads * ((self.vdim + 1) * self.dim + 1)

    def bind(self, num_blocks: int, block_size: int, num_slots: int, copies: int = 1) -> None:
        z = lambda *s: torch.zeros(*s, dtype=torch.float32, device=self.device)
        self.state = [z(num_slots, self.heads, self.vdim + 1, self.dim) for _ in range(copies)]
        self.m_state = [z(num_slots, self.heads) for _ in range(copies)]

    def unbind(self) -> None:
        self.state, self.m_state = [], []

    def rotations(self):
        return []

    def _gate_inputs(self, h: torch.Tensor) -> torch.Tensor:
        if self._mm_f32_out:
            try:
                return torch.mm(h, self.w_if.t(), out_dtype=torch.float32)
            except (RuntimeError, TypeError):
                self._mm_f32_out = False
        return F.linear(h, self.w_if).float()

    def mix(self, proj: torch.Tensor, h: torch.Tensor, positions, ctx, spans: mixops.StepSpans, inst: int, out: torch.Tensor | None = None,
            out_scale: float = 1.0) -> torch.Tensor:
        """proj [n, in_cols] = h W_in^T (a row-strided view) -> the output projection's operand [n, heads * vdim]."""
        Q, V = self.qk_cols, self.v_cols
        log_decay, write, floor = mixops.mlstm_gates(self._gate_inputs(h), self.b_if, self.cap, self.m_state[inst], ctx.state_slots, spans, self.heads)
        o = mixops.linear_state(proj, 0, Q, 2 * Q, self.state[inst], ctx.state_slots, spans, self.heads, self.heads, self.dim, self.vdim,
                                self.dim ** -0.5, log_decay=log_decay, write=write, ones=True)
        return mixops.head_rmsnorm_gate(o, self.norm_w, proj[:, 2 * Q + V:], self.eps, self.dtype, silu=False, out=out, out_scale=out_scale, floor=floor)

    def forward(self, h: torch.Tensor, positions, ctx, spans: mixops.StepSpans, inst: int = 0) -> torch.Tensor:
        return F.linear(self.mix(F.linear(h, self.w_in), h, positions, ctx, spans, inst), self.w_o)
