"""ncu target: one launch each (after one warm-up each) of the two head-decay recurrences and of the 16-bit prefill
attention over a window and pooled blocks, 4 x 2048-token prompts.
usage: python scripts/prof_fudonex.py"""
import sys

import torch

sys.path.insert(0, ".")
from semi_pd_b200 import ops  # noqa: E402

dev, bf = torch.device("cuda:0"), torch.bfloat16
n_req, L = 4, 2048
T = n_req * L
torch.manual_seed(0)


def i32(v):
    return torch.tensor(v, dtype=torch.int32, device=dev)


def rand(*s):
    return torch.randn(*s, device=dev, dtype=bf)


ext = dict(prefix_lens=i32([0] * n_req), extend_lens=i32([L] * n_req), extend_start_loc=i32([r * L for r in range(n_req)]))
rpi = torch.arange(n_req, device=dev)


def recurrence(form, H, kh, dk, dv):
    state = torch.zeros(n_req + 1, H, dv, dk, device=dev)
    q, k, v, z, b = rand(T, kh * dk), rand(T, kh * dk), rand(T, H * dv), rand(T, H), rand(T, H)
    kw = dict(num_heads=H, num_k_heads=kh, head_dim=dk, v_dim=dv, form=form, dt_bias=torch.full((H,), -2.0, device=dev),
              a_log=torch.zeros(H, device=dev), skip=torch.ones(H, device=dev) if form == "ssd" else None,
              b=b if form == "delta" else None, **ext)
    return lambda: ops.head_decay_recurrence(q, k, v, z, state, rpi, **kw)


H, G, D, window, size, run = 16, 4, 128, 1024, 32, 128
base = (T // run + 2) * run + 1
k_pool, v_pool = (rand(base + (T // run + 2) * (run // size), G, D) for _ in range(2))
qa, sinks = rand(T, H * D), torch.zeros(H, device=dev)
r2t = (torch.arange(T, device=dev, dtype=torch.int32) + 1).view(n_req, L).contiguous()


def attention():
    ops.attn_general(qa, k_pool, v_pool, r2t, rpi, H, G, D, D, D ** -0.5, window=window, sinks=sinks,
                     blocks=(size, run, base), max_extend_len=L, **ext)


launches = [recurrence("delta", 16, 8, 128, 128), recurrence("ssd", 64, 1, 128, 64), attention]
for _ in range(2):  # the first pass warms up
    for f in launches:
        f()
torch.cuda.synchronize()
