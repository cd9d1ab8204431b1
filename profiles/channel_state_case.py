"""One small case of the channel-decay matrix-state kernels for an `ncu` capture: `python profiles/channel_state_case.py delta|gla prefill|decode`
(16 heads, 128 x 128 states: a 4 x 1024-token prompt step, or a single-token step of 64 sequences)."""
import os
import sys

import torch

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, os.path.join(ROOT, "nano-vllm_b200"))

from nanovllm import mixops  # noqa: E402

rule, step = sys.argv[1:3]
H, d, dev = 16, 128, "cuda"
G = 4 if rule == "delta" else H
S, q = (4, 1024) if step == "prefill" else (64, 1)
n = S * q
if q > 1:
    cu = torch.arange(0, S + 1, dtype=torch.int32, device=dev) * q
    sp = mixops.StepSpans(S, q, cu, cu, None)
else:
    sp = mixops.StepSpans(S, 1, None, None, torch.full((S,), 100, dtype=torch.int32, device=dev))
x = torch.randn(n, (2 * G + H) * d, device=dev).bfloat16()
write = torch.randn(n, H, device=dev).bfloat16() if rule == "delta" else None
rate, bias = -torch.rand(H, device=dev), torch.zeros(H * d, device=dev)
state = torch.zeros(S, H, d, d, device=dev)
slots = torch.arange(S, dtype=torch.int32, device=dev)
for _ in range(4):
    z = torch.randn(n, H * d, device=dev)
    o = mixops.channel_state(x, 0, G * d, 2 * G * d, write, z, rate, bias, 1.0, state, slots, sp, H, G, d, d, d ** -0.5)
torch.cuda.synchronize()
print("ok", float(o.abs().mean()))
