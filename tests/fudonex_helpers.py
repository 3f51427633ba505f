"""Configurations of the Fudonex tests (small sizes of their own, chosen to reach every kernel route).  Model folders,
trace sessions and the error measure are shared with tests/rimidra_helpers.py."""
from oracle import fudonex_oracle as F


def config_mixed():
    """All three mixers; grouped heads, a rotation of half the head with rescaled frequencies, windows and blocks shorter
    than the prompts; two layers that read the first layer's cache, one with another window and block size, one with a
    window alone; two groups and two norm parts in a state-space layer, layers without feed-forward."""
    yarn = (4.0, 60, 3.0, 0.5)
    return F.make_config([
        F.attention_spec(heads=4, kv_heads=2, dim=16, vdim=24, scale=0.6, window=12, pool=8, rot_dims=8, base=500.0,
                         scaling=yarn, ff=40),
        F.mamba2_spec(heads=4, vdim=24, state=16, groups=2, conv=3, norm_groups=2, ff=48),
        F.attention_spec(heads=6, kv_heads=2, dim=16, vdim=24, scale=0.5, window=20, pool=5, rot_dims=8, base=500.0,
                         scaling=yarn, kv_from=0),
        F.delta_spec(heads=4, kv_heads=2, dim=16, vdim=8, conv=4, ff=32),
        F.attention_spec(heads=2, kv_heads=2, dim=16, vdim=24, scale=0.5, window=9, rot_dims=8, base=500.0, scaling=yarn,
                         kv_from=0, ff=24),
        F.attention_spec(heads=3, kv_heads=1, dim=24, vdim=16, scale=0.4, window=30, pool=4, rot_dims=24, base=90.0, ff=56),
    ], width=64, vocab=96, embed_scale=5.0, residual_mult=0.6, softcap=9.0)


def config_ones():
    """What a usual model makes > 1 is 1 or absent here: one head, windows of one token, blocks of one and of two tokens,
    one tap, one group, states of one row, no rotation, no scaling, multipliers 1, no cap on the logits, no feed-forward
    in some layers; sizes off the multiples of 4 and 8 (element-wise kernels and CUDA-core GEMMs even in 16 bits).  The
    norms run over a handful of channels, so their eps is large enough to keep rounding from being amplified."""
    return F.make_config([
        F.attention_spec(heads=1, kv_heads=1, dim=10, vdim=6, scale=1.0, window=1, pool=1, ff=10),
        F.mamba2_spec(heads=1, vdim=7, state=1, groups=1, conv=1, norm_groups=1),
        F.delta_spec(heads=1, kv_heads=1, dim=11, vdim=5, conv=1, ff=14),
        F.attention_spec(heads=3, kv_heads=3, dim=6, vdim=5, scale=0.7, window=1, pool=2, rot_dims=2, base=30.0),
        F.mamba2_spec(heads=3, vdim=5, state=9, groups=3, conv=2, norm_groups=5, ff=9),
        F.delta_spec(heads=2, kv_heads=1, dim=7, vdim=3, conv=2),
        F.attention_spec(heads=2, kv_heads=1, dim=4, vdim=4, scale=0.5, ff=6),
    ], width=36, vocab=50, eps=0.05)


def config_wide():
    """Shapes that the tensor-core GEMMs and attention kernels tile (64 / 64, 128 / 64), groups of 4 query heads, a window
    that crosses the cache's run length, blocks that divide a run; key sizes of the recurrences for each of the kernel's
    row counts (32, 64, 128, more)."""
    yarn = (8.0, 100, 4.0, 1.0)
    return F.make_config([
        F.attention_spec(heads=8, kv_heads=2, dim=64, vdim=64, scale=0.3, window=40, pool=16, rot_dims=64, base=3e4,
                         scaling=yarn, ff=192),
        F.mamba2_spec(heads=6, vdim=32, state=64, groups=3, conv=4, norm_groups=3, ff=128),
        F.delta_spec(heads=4, kv_heads=2, dim=128, vdim=64, conv=4, ff=128),
        F.attention_spec(heads=4, kv_heads=2, dim=64, vdim=64, scale=0.25, window=140, pool=32, rot_dims=64, base=3e4,
                         scaling=yarn, kv_from=0),
        F.attention_spec(heads=4, kv_heads=1, dim=128, vdim=64, scale=0.2, window=24, pool=64, rot_dims=32, base=1e4, ff=64),
        F.delta_spec(heads=2, kv_heads=2, dim=160, vdim=40, conv=3, ff=64),
        F.mamba2_spec(heads=2, vdim=96, state=24, groups=1, conv=8, norm_groups=1),
        F.delta_spec(heads=6, kv_heads=3, dim=32, vdim=48, conv=2),
    ], width=256, vocab=264, embed_scale=8.0, residual_mult=0.4, softcap=25.0)


def config_far():
    """Sharp scores (every query looks at one key or block, wherever it is), blocks of three tokens and states that hardly
    forget (weights of `far_weights`): what the first tokens say reaches any position."""
    return F.make_config([
        F.attention_spec(heads=2, kv_heads=1, dim=16, vdim=16, scale=1.5, window=7, pool=3, rot_dims=4, base=50.0),
        F.delta_spec(heads=2, kv_heads=2, dim=8, vdim=16, conv=2),
        F.mamba2_spec(heads=2, vdim=8, state=16, groups=1, conv=2, norm_groups=1, ff=24),
        F.attention_spec(heads=2, kv_heads=1, dim=16, vdim=16, scale=1.5, window=33, pool=11, rot_dims=4, base=50.0,
                         kv_from=0, ff=16),
    ], width=32, vocab=64)


def far_weights(cfg, seed):
    W = F.random_weights(cfg, seed)
    for name in W:
        if name.endswith("A_log"):
            W[name] = W[name] * 0 - 7.0
        if name.endswith("mix.sink"):
            W[name] = W[name] - 2.0
    return W


def config_uneven():
    """Sizes in whole 16-byte vectors that no attention tile fits; blocks that do not divide a run (48) and blocks longer
    than one (200); a window of exactly a run; three query heads per key head; a key size of three quarters of a row
    count; values wider and narrower than keys."""
    return F.make_config([
        F.attention_spec(heads=6, kv_heads=2, dim=40, vdim=80, scale=0.3, window=128, pool=48, rot_dims=24, base=7e3, ff=88),
        F.delta_spec(heads=3, kv_heads=1, dim=48, vdim=80, conv=4, ff=40),
        F.attention_spec(heads=2, kv_heads=2, dim=40, vdim=80, scale=0.3, window=17, pool=200, rot_dims=24, base=7e3,
                         kv_from=0),
        F.mamba2_spec(heads=5, vdim=40, state=96, groups=5, conv=5, norm_groups=10, ff=72),
    ], width=192, vocab=300, embed_scale=2.5, residual_mult=0.8, softcap=40.0)


CONFIGS = {"mixed": config_mixed, "ones": config_ones, "wide": config_wide, "far": config_far, "uneven": config_uneven}
SEEDS = {"mixed": 5, "ones": 12, "wide": 8, "far": 4, "uneven": 6}


def make_weights(name, cfg):
    return far_weights(cfg, SEEDS[name]) if name == "far" else F.random_weights(cfg, SEEDS[name])
