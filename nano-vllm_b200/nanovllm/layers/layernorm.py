"""RMSNorm module (reference nanovllm/layers/layernorm.py:5-50) on the CUDA kernels."""
from __future__ import annotations

import torch
from torch import nn

from .. import ops


class RMSNorm(nn.Module):
    def __init__(self, hidden_size: int, eps: float = 1e-6):
        super().__init__()
        self.eps = eps
        self.weight = nn.Parameter(torch.ones(hidden_size), requires_grad=False)

    def forward(self, x: torch.Tensor, residual: torch.Tensor | None = None):
        """``norm(x)``, or ``(norm(x + residual), bf16(x + residual))`` when a residual is given.

        The fused form updates ``residual`` in place and returns it (the reference returns a new tensor
        with the same values)."""
        if residual is None:
            return ops.rmsnorm(x, self.weight, self.eps)
        return ops.add_rmsnorm(x, residual, self.weight, self.eps)


class ResidualLayerNorm:
    """Weight-only layer norm reading an fp32 residual stream, fused with the stream's update: ``x += a + b`` (the two
    branches of a parallel block, summed first), then ``(x - mean) / sqrt(var + eps) * w`` in the model's activation type.
    A plain object (no nn.Module): ``weight`` is a device tensor set by the model's loader."""

    def __init__(self, width: int, eps: float, dtype, device):
        self.eps = eps
        self.weight = torch.ones(width, dtype=dtype, device=device)

    def __call__(self, x, a=None, b=None, b32=None, rows_idx=None):
        from .. import mixops
        return mixops.add_layernorm(x, self.weight, self.eps, a=a, b=b, b32=b32, rows_idx=rows_idx)


class SublayerOutputNorm:
    """RMS norm on a sublayer's OUTPUT with a weight stored around zero, fused with the scaled residual update of an fp32
    stream: ``x += mult * y / sqrt(mean(y^2) + eps) * (1 + w)``.  ``copy`` receives the updated rows in the activation type
    (the next sublayer's GEMM operand; the sublayers read the stream itself, not a normed copy)."""

    def __init__(self, width: int, eps: float, dtype, device):
        self.eps = eps
        self.weight = torch.zeros(width, dtype=dtype, device=device)

    def __call__(self, x, y, mult: float, copy=None) -> None:
        from .. import mixops
        mixops.add_normed(x, y, self.weight, mult, self.eps, w_offset=1.0, copy=copy)


class SandwichNorm:
    """The norms around one sublayer of a block that norms a sublayer on both sides, ``x <- x + norm_out(f(norm_in(x)))``, both RMS norms
    with weights stored around zero (``x / sqrt(mean(x^2) + eps) * (1 + w)``) over an fp32 stream.  ``open`` norms the stream
    for the sublayer; ``close`` norms the sublayer's output, updates the stream and, given the sublayer that follows, opens
    that one in the same pass (``copy``: the updated rows in the activation type instead, for a consumer that reads the stream itself)."""

    def __init__(self, width: int, eps: float, dtype, device):
        self.eps = eps
        self.w_in = torch.zeros(width, dtype=dtype, device=device)
        self.w_out = torch.zeros(width, dtype=dtype, device=device)

    def open(self, x):
        from .. import mixops
        return mixops.rmsnorm_rows(x, self.w_in, self.eps, w_offset=1.0)

    def close(self, x, y, then: "SandwichNorm | None" = None, copy=None):
        from .. import mixops
        return mixops.add_normed_norm(x, y, self.w_out, self.eps, w_offset=1.0, next_weight=then.w_in if then is not None else None,
                                      next_offset=1.0, copy=copy)


class GatedScaledSandwich:
    """The norms, gate and column scale around one sublayer of a block that reads a normed stream and gates, norms and scales the
    sublayer's result:

        h = rms(x) * g_in                          (g_in, g_out: ONE number each)
        x <- x + ls * rms(f(h) * sigmoid(W_r h + b_r)) * g_out

    over an fp32 stream.  The gate's pre-activation ``W_r h + b_r`` comes from the sublayer (its rows ride in the sublayer's input
    projection, which reads the same h).  ``g_out * ls`` is folded into one fp32 vector when either is loaded; ``g_in`` is kept as a
    vector in the activation type (the opening norm of a step) and in fp32 (the opening norm fused into the previous close)."""

    def __init__(self, width: int, eps: float, dtype, device):
        self.eps, self.dtype = eps, dtype
        self.g_out = torch.ones(1, dtype=torch.float32, device=device)
        self.ls = torch.ones(width, dtype=torch.float32, device=device)
        self.w_out = torch.ones(width, dtype=torch.float32, device=device)        # g_out * ls
        self.w_in32 = torch.ones(width, dtype=torch.float32, device=device)       # g_in on every column
        self.w_in = torch.ones(width, dtype=dtype, device=device)

    def load(self, which: str, w: torch.Tensor) -> None:
        w = w.to(self.w_out.device, torch.float32).reshape(-1)
        if which == "in":
            self.w_in32.copy_(w.expand_as(self.w_in32))
            self.w_in.copy_(self.w_in32)
            return
        if which == "out":
            self.g_out.copy_(w)
        else:
            self.ls.copy_(w)
        torch.mul(self.ls, self.g_out, out=self.w_out)

    def open(self, x):
        from .. import mixops
        return mixops.rmsnorm_rows(x, self.w_in, self.eps)

    def close(self, x, y, gate, then: "GatedScaledSandwich | None" = None):
        """x += ls * norm_out(y * sigmoid(gate)); with ``then`` also returns that sublayer's normed input."""
        from .. import mixops
        return mixops.gated_add_normed_norm(x, y, gate, self.w_out, self.eps, self.dtype, next_scale=1.0 if then is not None else None,
                                            w_next=then.w_in32 if then is not None else None)


class PreNorm:
    """The RMS norm in front of one sublayer of a pre-norm layer, ``x <- x + f(rms(x) * w)`` over an fp32 stream.  ``after`` closes the sublayer
    before it (``x += y``) in the same pass; ``scale`` is a constant factor on the result."""

    def __init__(self, width: int, eps: float, dtype, device, scale: float = 1.0):
        self.eps, self.scale = eps, scale
        self.weight = torch.ones(width, dtype=dtype, device=device)

    def open(self, x, rows_idx=None):
        """The norm of the stream (of the rows ``rows_idx``)."""
        from .. import mixops
        return mixops.add_rmsnorm(x, self.weight, self.eps, rows_idx=rows_idx, out_scale=self.scale)

    def after(self, x, y):
        """x += y in place; returns the norm of the result."""
        from .. import mixops
        return mixops.add_rmsnorm(x, self.weight, self.eps, y=y, out_scale=self.scale)


class ParallelNorms:
    """The two biased layer norms of a parallel block, ``x <- x + m (f1(ln1(x)) + f2(ln2(x)))`` over an fp32 stream: both read the same x,
    so one pass forms the statistics once and writes both results.  ``advance`` closes a block (the scaled update with the summed
    branches, then optionally another fp32 stream added on top) and opens the next one in the same pass.  ``second=False``: a block
    with one branch."""

    def __init__(self, width: int, eps: float, dtype, device, second: bool = True):
        self.eps = eps
        self.norm1 = (torch.ones(width, dtype=dtype, device=device), torch.zeros(width, dtype=dtype, device=device))
        self.norm2 = (torch.ones(width, dtype=dtype, device=device), torch.zeros(width, dtype=dtype, device=device)) if second else None

    def load(self, leaf: str, w: torch.Tensor) -> bool:
        named = {"norm1": self.norm1[0], "norm1.b": self.norm1[1]}
        if self.norm2 is not None:
            named.update({"norm2": self.norm2[0], "norm2.b": self.norm2[1]})
        if leaf not in named:
            return False
        named[leaf].copy_(w)
        return True

    def weight_shapes(self, width: int) -> dict:
        return {k: (width,) for k in ("norm1", "norm1.b") + (("norm2", "norm2.b") if self.norm2 is not None else ())}

    def open(self, x, add=None, rows_idx=None):
        """(ln1(x), ln2(x) or None) after ``x += add``."""
        from .. import mixops
        return mixops.add_layernorm2(x, self.eps, add=add, norm1=self.norm1, norm2=self.norm2, rows_idx=rows_idx)

    def advance(self, x, y, mult: float, then: "ParallelNorms | None" = None, add=None, x_out=None):
        """x_out (None: x itself) = x + mult * y + add; with ``then`` also that block's (ln1, ln2) of the result."""
        from .. import mixops
        return mixops.add_layernorm2(x, self.eps, y=y, mult=mult, add=add, x_out=x_out, norm1=then.norm1 if then is not None else None,
                                     norm2=then.norm2 if then is not None else None)
