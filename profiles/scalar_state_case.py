"""One small case of the scalar linear-attention kernels for an `ncu` capture: `python profiles/scalar_state_case.py space|memory prefill|decode`
(state space: 32 heads of 64 x 128 over 4 groups; matrix memory: 16 heads of 128 x 128; an 8 x 1024-token prompt step, or a single-token
step of 64 sequences)."""
import os
import sys

import torch

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, os.path.join(ROOT, "nano-vllm_b200"))

from nanovllm import mixops  # noqa: E402

rule, step = sys.argv[1:3]
d, dev = 128, "cuda"
S, q = (8, 1024) if step == "prefill" else (64, 1)
n = S * q
if q > 1:
    cu = torch.arange(0, S + 1, dtype=torch.int32, device=dev) * q
    sp = mixops.StepSpans(S, q, cu, cu, None)
else:
    sp = mixops.StepSpans(S, 1, None, None, torch.full((S,), 100, dtype=torch.int32, device=dev))
slots = torch.arange(S, dtype=torch.int32, device=dev)
if rule == "space":
    H, G, vd = 32, 4, 64
    x, dt = torch.randn(n, H * vd + 2 * G * d, device=dev).bfloat16(), torch.randn(n, H, device=dev).bfloat16()
    state, rate, bias = torch.zeros(S, H, vd, d, device=dev), -torch.rand(H, device=dev), torch.zeros(H, device=dev)
    run = lambda: mixops.linear_state(x, H * vd + G * d, H * vd, 0, state, slots, sp, H, G, d, vd, step=dt, rate=rate, bias=bias)
else:
    H = 16
    x, ld, w = torch.randn(n, 3 * H * d, device=dev).bfloat16(), -torch.rand(n, H, device=dev), torch.rand(n, H, device=dev)
    state = torch.zeros(S, H, d + 1, d, device=dev)
    run = lambda: mixops.linear_state(x, 0, H * d, 2 * H * d, state, slots, sp, H, H, d, d, d ** -0.5, log_decay=ld, write=w, ones=True)
for _ in range(4):
    o = run()
torch.cuda.synchronize()
print("ok", float(o.abs().mean()))
