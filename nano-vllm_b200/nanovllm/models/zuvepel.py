"""Zuvepel: a decoder of parallel layers with two layer norms, ``x <- x + m (mixer(ln1(x)) + ff(ln2(x)))``, biased norms, the token
embedding scaled by a constant.  The mixer of a layer is chunked grouped-query attention with a softmax sink and a gate per head
(``attention``), a delta rule with a decay per key channel (``channel_delta``) or gated linear attention (``gla``); the feed-forward is
a gated dense block, or absent.  A run of consecutive layers may be repeated several times with the same weights; every repetition
(pass) but the first opens with ``x <- x + x0`` (x0: the embedding output) and has caches and states of its own.  config.json
(``"architecture": "Zuvepel"``) lists the layers and gives every constant; the ranks of the low-rank maps come from the tensors.

The residual stream is fp32 in both number formats; projections, caches and branch outputs are bf16 (serving) or fp32; what
enters a recurrence, attention statistics and norms are fp32 in both.  Like the other models of this package it is a plain
object: named device tensors and a flat list of launches per step, the same for prompt portions, mixed batches and (captured in
CUDA graphs) decode steps.

Cache and state: per attention mixer and pass a paged key/value cache (``[blocks * block_size, kv_heads * (dim + vdim)]``,
addressed through the engine's block tables and slot numbers); per recurrent mixer and pass a state slot per live sequence
(matrix state and, for the delta rule, convolution history).  The engine's block manager hands out pages and slots.
"""
from __future__ import annotations

import torch
import torch.nn.functional as F

from .. import mixops
from ..layers.channel_state import ChannelDeltaMixer, GatedLinearAttention
from ..layers.layernorm import ParallelNorms
from ..layers.parallel_block import ParallelBranches
from ..layers.window_attention import ChunkedSinkAttention
from ..utils.context import get_context
from .layer_order import layer_runs

MIXERS = {"attention": ChunkedSinkAttention, "channel_delta": ChannelDeltaMixer, "gla": GatedLinearAttention}


class ZuvepelConfig:
    """The parsed config.json plus the attribute names the engine reads from any model configuration."""
    architectures = ["Zuvepel"]

    def __init__(self, raw: dict, max_position_embeddings: int = 1 << 20):
        self.raw = raw
        self.layers = raw["layers"]
        self.vocab_size = int(raw["vocab"])
        self.hidden_size = int(raw["width"])
        self.norm_eps = float(raw["norm"]["eps"])
        self.embed_scale = float((raw.get("embedding") or {}).get("scale", 1.0))
        self.residual_mult = float(raw.get("residual_mult", 1.0))
        self.loop = raw.get("loop") or None
        self.num_hidden_layers = len(self.layers)
        self.max_position_embeddings = int(raw.get("max_position", max_position_embeddings))
        self.eos_token_id = raw.get("eos")
        # (layer, pass, whether the embedding output is added right before it)
        self.runs = [(i, k, opens and k > 0) for i, k, opens in layer_runs(len(self.layers), self.loop)]
        for i, layer in enumerate(self.layers):
            if layer["type"] not in MIXERS:
                raise ValueError(f"layer {i}: unknown mixer type {layer['type']!r}")
            mlp = layer.get("mlp")
            if mlp is not None and mlp.get("kind") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")

    def passes_of(self, layer: int) -> int:
        return max(k for i, k, _ in self.runs if i == layer) + 1


class _Block:
    __slots__ = ("norms", "branches", "passes")


class ZuvepelForCausalLM:
    needs_block_tables = True        # attention always reads keys through the block tables, also in a first portion
    zero_centred = ()

    def __init__(self, hf_config: ZuvepelConfig, tp_rank: int = 0, tp_size: int = 1, device="cuda", max_position: int | None = None,
                 dtype=torch.bfloat16):
        if tp_size != 1:
            raise NotImplementedError("Zuvepel runs on one GPU (no tensor-parallel sharding of its mixers yet)")
        c = hf_config
        self.cfg, self.device, self.dtype = c, torch.device(device), dtype
        self.hidden, self.eps = c.hidden_size, c.norm_eps
        self.vocab_shard = c.vocab_size
        self.tp_rank, self.tp_size = tp_rank, tp_size
        max_position = int(max_position or c.max_position_embeddings)
        W = self.hidden
        e = lambda *s: torch.empty(*s, dtype=dtype, device=self.device)
        self.embed, self.lm_head = e(c.vocab_size, W), e(c.vocab_size, W)
        self.final = ParallelNorms(W, self.eps, dtype, self.device, second=False)
        self.blocks: list[_Block] = []
        tables: dict = {}
        for i, layer in enumerate(c.layers):
            b = _Block()
            b.passes = c.passes_of(i)
            mlp = layer.get("mlp")
            b.norms = ParallelNorms(W, self.eps, dtype, self.device, second=mlp is not None)
            extra = dict(max_position=max_position) if layer["type"] == "attention" else {}
            b.branches = ParallelBranches(W, MIXERS[layer["type"]], layer["mixer"], mlp, dtype, self.device, eps=self.eps, **extra)
            if layer["type"] == "attention" and b.branches.mixer.cos_sin is not None:
                att = b.branches.mixer
                att.cos_sin = tables.setdefault(att.rot_key, att.cos_sin)               # layers with one rotation share its table
            self.blocks.append(b)
        self.has_recurrent_state = any(layer["type"] != "attention" for layer in c.layers)
        # a cached prefix can be skipped only when all that remembers it is in the pages
        self.supports_prefix_cache = not self.has_recurrent_state
        self.block_size = 0
        self._bound = False
        self._mm_f32_out = True

    # ---- weights -----------------------------------------------------------------------------------------------------
    def declare_shapes(self, shapes: dict) -> None:
        """Tensor shapes of the checkpoint about to be loaded: the low-rank maps take their ranks from them."""
        for i, b in enumerate(self.blocks):
            m = b.branches.mixer
            if hasattr(m, "set_ranks"):
                m.set_ranks({leaf: shapes[f"l{i}.mix.{leaf}"][0] for leaf, _ in m.low_rank() if f"l{i}.mix.{leaf}" in shapes})

    def load_hf_tensor(self, name: str, w: torch.Tensor) -> None:
        """Place one checkpoint tensor: ``embed``, ``head``, ``final.norm[.b]``, ``l<i>.norm1|norm2[.b]``, ``l<i>.mix.<leaf>``,
        ``l<i>.mlp.<leaf>``."""
        top = {"embed": self.embed, "head": self.lm_head, "final.norm": self.final.norm1[0], "final.norm.b": self.final.norm1[1]}
        if name in top:
            top[name].copy_(w)
            return
        head, _, rest = name.partition(".")
        if not (head.startswith("l") and head[1:].isdigit()) or int(head[1:]) >= len(self.blocks):
            raise KeyError(f"unexpected checkpoint tensor {name}")
        b = self.blocks[int(head[1:])]
        if rest.startswith("mix."):
            ok = b.branches.mixer.load(rest[4:], w)
        elif rest.startswith("mlp."):
            ok = b.branches.ff is not None and b.branches.ff.load(rest[4:], w)
        else:
            ok = b.norms.load(rest, w) or (b.norms.norm2 is None and rest in ("norm2", "norm2.b"))     # no feed-forward: nothing reads them
        if not ok:
            raise KeyError(f"unexpected checkpoint tensor {name}")

    def weight_shapes(self) -> dict:
        """name -> shape of every checkpoint tensor of this configuration (random initialisation, tests)."""
        c, W = self.cfg, self.hidden
        out = {"embed": (c.vocab_size, W), "head": (c.vocab_size, W), "final.norm": (W,), "final.norm.b": (W,)}
        for i, b in enumerate(self.blocks):
            p = f"l{i}."
            out.update({p + k: v for k, v in b.norms.weight_shapes(W).items()})
            out.update({p + "mix." + k: v for k, v in b.branches.mixer.weight_shapes(W).items()})
            if b.branches.ff is not None:
                out.update({p + "mlp." + k: v for k, v in b.branches.ff.weight_shapes(W).items()})
        return out

    # ---- cache and state ---------------------------------------------------------------------------------------------
    def cache_block_bytes(self, block_size: int) -> int:
        elem = 4 if self.dtype == torch.float32 else 2
        return sum(b.branches.mixer.cache_row_elems() * b.passes for b in self.blocks) * block_size * elem

    def state_slot_bytes(self) -> int:
        return sum(b.branches.mixer.state_slot_bytes() * b.passes for b in self.blocks)

    def bind_cache(self, num_blocks: int, block_size: int, num_state_slots: int) -> None:
        self.block_size = block_size
        for b in self.blocks:
            b.branches.mixer.bind(num_blocks, block_size, max(num_state_slots, 1), b.passes)
        self._bound = True

    def unbind_cache(self) -> None:
        for b in self.blocks:
            b.branches.mixer.unbind()
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
        after every layer run, before the embedding output that opens a next pass is added."""
        if not self._bound:
            raise RuntimeError("bind_cache() first: this model has no cache-less path")
        ctx, c = get_context(), self.cfg
        spans = self._spans(ctx, input_ids.shape[0])
        runs = c.runs
        x0 = mixops.embed_pair(input_ids, self.embed, c.embed_scale, spans)
        keep_x0 = any(reopens for _, _, reopens in runs)
        x = x0
        h1, h2 = self.blocks[runs[0][0]].norms.open(x)
        for r, (i, k, _) in enumerate(runs):
            b = self.blocks[i]
            y = b.branches.forward(h1, h2, positions, ctx, spans, k)
            nxt = runs[r + 1] if r + 1 < len(runs) else None
            then = self.blocks[nxt[0]].norms if nxt is not None else None
            add = x0 if nxt is not None and nxt[2] else None
            x_out = torch.empty_like(x) if keep_x0 and x is x0 else x
            if taps is None:
                h1, h2 = b.norms.advance(x, y, c.residual_mult, then, add, x_out)
                x = x_out
            else:
                b.norms.advance(x, y, c.residual_mult, x_out=x_out)
                x = x_out
                taps.append(x.clone())
                if then is not None:
                    h1, h2 = then.open(x, add)
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
        hn, _ = self.final.open(hidden, rows_idx=rows)
        if self.dtype == torch.float32:
            return F.linear(hn, self.lm_head)
        if self._mm_f32_out:
            try:
                return torch.mm(hn, self.lm_head.t(), out_dtype=torch.float32)        # bf16 operands, fp32 accumulator written as is
            except (RuntimeError, TypeError):
                self._mm_f32_out = False          # shapes or a library build without that output type: round once to bf16 instead
        return F.linear(hn, self.lm_head).float()
