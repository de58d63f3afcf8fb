"""One recurrence launch sequence on a small case, for a profiler: decode | chunk (time-mix mode)."""
import os
import sys

import torch

sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
from benchmarks.mixer_bench import batch, rnd  # noqa: E402
from metrale_inference_alpha_b200.ops import check_status, mixers as mx  # noqa: E402

case = sys.argv[1]
H, D = 20, 128
lens, start = ([1] * 128, 63) if case == "decode" else ([4096], 0)
b, _ = batch(lens, start)
T = sum(lens)
q, k, v = (rnd(T, H * D) for _ in range(3))
lw, u = -torch.exp(torch.randn(T, H * D, device="cuda") - 3), torch.rand(H, D, device="cuda")
ssm = torch.zeros(len(lens) + 2, H, D, D, device="cuda")
for _ in range(3):
    mx.linear_attention(q, k, v, ssm, b, heads=H, dk=D, dv=D, fmt="bf16", log_w=lw, u=u)
torch.cuda.synchronize()
check_status("cuda")
