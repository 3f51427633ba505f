"""ncu target: one launch each (after one warm-up each) of the rotary step with a norm over the whole row and of the 16-bit
prefill attention over a window alone, with kept first tokens and with a distance table, 4 x 2048-token prompts.
usage: python scripts/prof_kuforax.py"""
import sys

import torch

sys.path.insert(0, ".")
from semi_pd_b200 import ops  # noqa: E402
from semi_pd_b200.kuforax import distance_buckets  # noqa: E402
from semi_pd_b200.matepel import scaled_rotary_table  # noqa: E402

dev, bf = torch.device("cuda:0"), torch.bfloat16
n_req, L = 4, 2048
T = n_req * L
H, G, D, window = 16, 4, 128, 1024
torch.manual_seed(0)


def i32(v):
    return torch.tensor(v, dtype=torch.int32, device=dev)


def rand(*s):
    return torch.randn(*s, device=dev, dtype=bf)


ext = dict(prefix_lens=i32([0] * n_req), extend_lens=i32([L] * n_req), extend_start_loc=i32([r * L for r in range(n_req)]))
rpi = torch.arange(n_req, device=dev)
k_pool, v_pool, q = rand(T + 128, G, D), rand(T + 128, G, D), rand(T, H * D)
r2t = (torch.arange(T, device=dev, dtype=torch.int32) + 1).view(n_req, L).contiguous()
table = torch.randn(32, H, device=dev)[torch.tensor(distance_buckets(32, window // 2, window), device=dev)].T.contiguous()


def attention(**kw):
    return lambda: ops.attn_general(q, k_pool, v_pool, r2t, rpi, H, G, D, D, D ** -0.5, window=window, max_extend_len=L, **ext, **kw)


y = rand(T, (H + G) * D + H)
qs, ks = y[:, : (H + G) * D].split([H * D, G * D], -1)
cs = scaled_rotary_table(D // 2, 1e6, None, L + 64, dev)
pos, loc = torch.arange(T, device=dev) % L, torch.randperm(T, device=dev) + 1
q_out, kf, vf = torch.empty(T, H * D, device=dev, dtype=bf), k_pool.view(-1, G * D), v_pool.view(-1, G * D)
ones = torch.ones(H * D, device=dev)
segments = [ops.rotary_segment(qs, q_out, H, D, D // 2, norm_eps=1e-6, norm_weight=ones, norm_row=True),
            ops.rotary_segment(ks, kf, G, D, D // 2, to_pool=True, norm_eps=1e-6, norm_weight=ones[: G * D], norm_row=True),
            ops.rotary_segment(ks, vf, G, D, 0, to_pool=True)]

launches = [lambda: ops.rotary_segments(segments, pos, cs, bf, loc=loc), attention(), attention(keep_first=4),
            attention(dist_bias=table)]
for _ in range(2):  # the first pass warms up
    for f in launches:
        f()
torch.cuda.synchronize()
