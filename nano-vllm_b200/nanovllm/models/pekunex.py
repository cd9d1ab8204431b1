"""Pekunex: a pre-norm decoder, ``x <- x + mixer(rms(x) w1)``, ``x <- x + ff(rms(x) w2)``, the token embedding scaled by a constant.  The mixer of
a layer is grouped-query attention with biases, unit-RMS queries and keys after a half-split rotation, soft-capped scores and an output
gate per element (``attention``); attention with a learned softmax sink beside a matrix memory with exponential gates, summed with two
constants (``parallel``); or a state-space recurrence with one decay per head and its gate before a grouped norm (``mamba2``).  The
feed-forward is a SiLU-gated dense block, or absent.  A layer may run with another layer's weights (``weights_of``) and a cache or state of
its own.  The logits carry a constant factor.  config.json (``"architecture": "Pekunex"``) lists the layers and gives every size and constant.

The residual stream is fp32 in both number formats; projections, convolution results, caches and branch outputs are bf16 (serving) or
fp32; norms, attention statistics, rotation angles and whatever enters a recurrence besides those are fp32 in both.  Like the other
models of this package it is a plain object: named device tensors and a flat list of launches per step, the same for prompt portions,
mixed batches and (captured in CUDA graphs) decode steps.

Cache and state: per attention (also the one inside a ``parallel`` layer) and layer run a paged cache ``[blocks * block_size, kv_heads *
(dim + vdim)]``, addressed through the engine's block tables and slot numbers; per recurrence and layer run a state slot per live
sequence.  The engine's block manager hands out pages and slots.
"""
from __future__ import annotations

import torch
import torch.nn.functional as F

from .. import mixops
from ..layers.layernorm import PreNorm
from ..layers.moe import SiluGatedDenseFF
from ..layers.parallel_mixer import ParallelMixer
from ..layers.scalar_state import MatrixMemoryMixer, StateSpaceMixer
from ..layers.window_attention import CappedGatedAttention, LearnedSinkAttention
from ..utils.context import get_context


def _parallel(width: int, m: dict, eps: float, dtype, device, max_position: int) -> ParallelMixer:
    return ParallelMixer(width, LearnedSinkAttention, m["left"], MatrixMemoryMixer, m["right"], m["left_scale"], m["right_scale"], dtype, device,
                         eps=eps, max_position=max_position)


MIXERS = {"attention": CappedGatedAttention, "parallel": _parallel, "mamba2": StateSpaceMixer}


class PekunexConfig:
    """The parsed config.json plus the attribute names the engine reads from any model configuration."""
    architectures = ["Pekunex"]

    def __init__(self, raw: dict, max_position_embeddings: int = 1 << 20):
        self.raw = raw
        self.layers = raw["layers"]
        self.vocab_size = int(raw["vocab"])
        self.hidden_size = int(raw["width"])
        self.norm_eps = float(raw["norm"]["eps"])
        self.embed_scale = float((raw.get("embedding") or {}).get("scale", 1.0))
        self.logit_scale = float(raw.get("logit_scale", 1.0))
        self.num_hidden_layers = len(self.layers)
        self.max_position_embeddings = int(raw.get("max_position", max_position_embeddings))
        self.eos_token_id = raw.get("eos")
        # runs: (layer that owns the weights, which of that layer's caches and states) in execution order
        self.runs: list[tuple[int, int]] = []
        self.copies: dict[int, int] = {}                 # weight-owning layer -> caches / states it needs
        for i, layer in enumerate(self.layers):
            if layer["type"] not in MIXERS:
                raise ValueError(f"layer {i}: unknown mixer type {layer['type']!r}")
            mlp = layer.get("mlp")
            if mlp is not None and mlp.get("kind") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
            src = self.owner_of(i)
            if layer["type"] != self.layers[src]["type"]:
                raise ValueError(f"layer {i}: its mixer type differs from layer {src}, whose weights it uses")
            self.runs.append((src, self.copies.get(src, 0)))
            self.copies[src] = self.copies.get(src, 0) + 1

    def owner_of(self, i: int) -> int:
        """The layer whose tensors layer i runs with (through borrowers of borrowers)."""
        seen = {i}
        while self.layers[i].get("weights_of") is not None:
            i = int(self.layers[i]["weights_of"])
            if not 0 <= i < len(self.layers) or i in seen:
                raise ValueError(f"weights_of must lead to a layer with tensors of its own, not back or to {i}")
            seen.add(i)
        return i


class _Block:
    __slots__ = ("norm1", "mixer", "norm2", "ff")


class PekunexForCausalLM:
    needs_block_tables = True        # attention always reads keys through the block tables, also in a first portion
    zero_centred = ("dt_bias",)

    def __init__(self, hf_config: PekunexConfig, tp_rank: int = 0, tp_size: int = 1, device="cuda", max_position: int | None = None,
                 dtype=torch.bfloat16):
        if tp_size != 1:
            raise NotImplementedError("Pekunex runs on one GPU (no tensor-parallel sharding of its mixers yet)")
        c = hf_config
        self.cfg, self.device, self.dtype = c, torch.device(device), dtype
        self.hidden, self.eps = c.hidden_size, c.norm_eps
        self.vocab_shard = c.vocab_size
        self.tp_rank, self.tp_size = tp_rank, tp_size
        max_position = int(max_position or c.max_position_embeddings)
        W = self.hidden
        e = lambda *s: torch.empty(*s, dtype=dtype, device=self.device)
        self.embed, self.lm_head = e(c.vocab_size, W), e(c.vocab_size, W)
        self.final = PreNorm(W, self.eps, dtype, self.device, scale=c.logit_scale)       # the head is linear: its factor rides in the norm
        self.blocks: dict[int, _Block] = {}
        tables: dict = {}
        for i, layer in enumerate(c.layers):
            if c.owner_of(i) != i:
                continue
            b = _Block()
            b.norm1 = PreNorm(W, self.eps, dtype, self.device)
            b.mixer = MIXERS[layer["type"]](W, layer["mixer"], self.eps, dtype, self.device, max_position)
            for att in b.mixer.rotations():
                if att.cos_sin is not None:
                    att.cos_sin = tables.setdefault(att.rot_key, att.cos_sin)             # layers with one rotation share its table
            mlp = layer.get("mlp")
            b.ff = SiluGatedDenseFF(W, mlp, dtype, self.device) if mlp is not None else None
            b.norm2 = PreNorm(W, self.eps, dtype, self.device) if mlp is not None else None
            self.blocks[i] = b
        self.has_recurrent_state = any(b.mixer.state_slot_bytes() > 0 for b in self.blocks.values())
        # a cached prefix can be skipped only when all that remembers it is in the pages
        self.supports_prefix_cache = not self.has_recurrent_state
        self.block_size = 0
        self._bound = False
        self._mm_f32_out = True

    # ---- weights -----------------------------------------------------------------------------------------------------
    def load_hf_tensor(self, name: str, w: torch.Tensor) -> None:
        """Place one checkpoint tensor: ``embed``, ``head``, ``final.norm``, ``l<i>.norm1|norm2``, ``l<i>.mix.<leaf>``, ``l<i>.mlp.<leaf>``."""
        top = {"embed": self.embed, "head": self.lm_head, "final.norm": self.final.weight}
        if name in top:
            top[name].copy_(w)
            return
        head, _, rest = name.partition(".")
        if not (head.startswith("l") and head[1:].isdigit()) or int(head[1:]) not in self.blocks:
            raise KeyError(f"unexpected checkpoint tensor {name}")
        b = self.blocks[int(head[1:])]
        ok = True
        if rest == "norm1":
            b.norm1.weight.copy_(w)
        elif rest == "norm2":
            if b.norm2 is not None:                      # no feed-forward: nothing reads it
                b.norm2.weight.copy_(w)
        elif rest.startswith("mix."):
            ok = b.mixer.load(rest[4:], w)
        else:
            ok = rest.startswith("mlp.") and b.ff is not None and b.ff.load(rest[4:], w)
        if not ok:
            raise KeyError(f"unexpected checkpoint tensor {name}")

    def weight_shapes(self) -> dict:
        """name -> shape of every checkpoint tensor of this configuration (random initialisation, tests)."""
        c, W = self.cfg, self.hidden
        out = {"embed": (c.vocab_size, W), "head": (c.vocab_size, W), "final.norm": (W,)}
        for i, b in self.blocks.items():
            p = f"l{i}."
            out[p + "norm1"] = (W,)
            out.update({p + "mix." + k: v for k, v in b.mixer.weight_shapes(W).items()})
            if b.ff is not None:
                out[p + "norm2"] = (W,)
                out.update({p + "mlp." + k: v for k, v in b.ff.weight_shapes(W).items()})
        return out

    # ---- cache and state ---------------------------------------------------------------------------------------------
    def cache_block_bytes(self, block_size: int) -> int:
        elem = 4 if self.dtype == torch.float32 else 2
        return sum(b.mixer.cache_row_elems() * self.cfg.copies[i] for i, b in self.blocks.items()) * block_size * elem

    def state_slot_bytes(self) -> int:
        return sum(b.mixer.state_slot_bytes() * self.cfg.copies[i] for i, b in self.blocks.items())

    def bind_cache(self, num_blocks: int, block_size: int, num_state_slots: int) -> None:
        self.block_size = block_size
        for i, b in self.blocks.items():
            b.mixer.bind(num_blocks, block_size, max(num_state_slots, 1), self.cfg.copies[i])
        self._bound = True

    def unbind_cache(self) -> None:
        for b in self.blocks.values():
            b.mixer.unbind()
        self._bound = False

    def modules(self):
        return iter(())               # no paged-GQA attention operators of the first library: the cache is bound through bind_cache()

    # ---- forward ------------------------------------------------------------------------------------------------------
    @staticmethod
    def _spans(ctx, n: int) -> mixops.StepSpans:
        if ctx.is_prefill:
            return mixops.StepSpans(ctx.cu_seqlens_q.numel() - 1, int(ctx.max_seqlen_q), ctx.cu_seqlens_q, ctx.cu_seqlens_k, None)
        return mixops.StepSpans(n, 1, None, None, ctx.context_lens)

    @torch.inference_mode()
    def forward(self, input_ids: torch.Tensor, positions: torch.Tensor, taps: list | None = None) -> torch.Tensor:
        """-> the fp32 residual stream after the last layer, [tokens, width].  ``taps`` (a list) collects a copy of the stream
        after every layer."""
        if not self._bound:
            raise RuntimeError("bind_cache() first: this model has no cache-less path")
        ctx, c = get_context(), self.cfg
        spans = self._spans(ctx, input_ids.shape[0])
        x = mixops.embed_pair(input_ids, self.embed, c.embed_scale, spans)
        h = self.blocks[c.runs[0][0]].norm1.open(x) if c.runs else None
        for r, (i, inst) in enumerate(c.runs):
            b = self.blocks[i]
            y = b.mixer.forward(h, positions, ctx, spans, inst)
            if b.ff is not None:
                y, _ = b.ff.forward(b.norm2.after(x, y))
            if r + 1 < len(c.runs):
                h = self.blocks[c.runs[r + 1][0]].norm1.after(x, y)
            else:
                mixops.add_rmsnorm(x, None, self.eps, y=y)
            if taps is not None:
                taps.append(x.clone())
        return x

    __call__ = forward

    @torch.inference_mode()
    def last_token_rows(self, hidden: torch.Tensor) -> torch.Tensor:
        raise NotImplementedError("the fused LM head takes bf16 rows; this model normalises selected rows in compute_logits")

    @torch.inference_mode()
    def compute_logits(self, hidden: torch.Tensor) -> torch.Tensor:
        """fp32 logits of the step's last token per sequence, or of the rows named by ``ctx.logit_rows`` (int32)."""
        ctx = get_context()
        rows = getattr(ctx, "logit_rows", None)
        if rows is None and ctx.is_prefill:
            rows = (ctx.cu_seqlens_q[1:] - 1).to(torch.int32)
        hn = self.final.open(hidden, rows_idx=rows)
        if self.dtype == torch.float32:
            return F.linear(hn, self.lm_head)
        if self._mm_f32_out:
            try:
                return torch.mm(hn, self.lm_head.t(), out_dtype=torch.float32)        # bf16 operands, fp32 accumulator written as is
            except (RuntimeError, TypeError):
                self._mm_f32_out = False          # shapes or a library build without that output type: round once to bf16 instead
        return F.linear(hn, self.lm_head).float()
