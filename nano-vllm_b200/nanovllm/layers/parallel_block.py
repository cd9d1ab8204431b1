"""A parallel block's two branches, ``mixer(h1) + ff(h2)``, with one output projection: ``W_o a + W_down b = [W_o | W_down] [a ; b]``.

Each branch writes its operand into its columns of one buffer and holds its output weights as a view into the merged ones, so the
branches are summed in the GEMM's fp32 accumulator and rounded once.  Without a feed-forward the block is the mixer alone.
"""
from __future__ import annotations

import torch
import torch.nn.functional as F

from .. import mixops
from .moe import GatedDenseFF


class ParallelBranches:
    def __init__(self, width: int, mixer_cls, mixer_cfg: dict, mlp: dict | None, dtype, device, **mixer_args):
        self.dtype, self.device = dtype, device
        self.split = mixer_cls.operand_cols(mixer_cfg)
        ff = int(mlp["ff"]) if mlp is not None else 0
        self.w_out = torch.empty(width, self.split + ff, dtype=dtype, device=device)
        self.mixer = mixer_cls(width, mixer_cfg, dtype=dtype, device=device, w_o=self.w_out[:, :self.split], **mixer_args)
        self.ff = GatedDenseFF(width, mlp, dtype, device, w_down=self.w_out[:, self.split:]) if mlp is not None else None

    def forward(self, h1: torch.Tensor, h2: torch.Tensor | None, positions, ctx, spans: mixops.StepSpans, inst: int = 0) -> torch.Tensor:
        both = torch.empty(h1.shape[0], self.w_out.shape[1], dtype=self.dtype, device=self.device)
        self.mixer.mix(h1, positions, ctx, spans, inst, out=both[:, :self.split])
        if self.ff is not None:
            self.ff.hidden(h2, out=both[:, self.split:])
        return F.linear(both, self.w_out)
