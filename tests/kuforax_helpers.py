"""Configurations of the Kuforax tests (small sizes of their own, chosen to reach every kernel route).  Model folders,
trace sessions and the error measure are shared with tests/rimidra_helpers.py."""
from oracle import kuforax_oracle as K


def config_mixed():
    """Both mixers, the middle two looped twice, grouped heads 4 : 2, values wider than keys in one of them, a rotation of
    half the head with rescaled frequencies, windows shorter than the prompts, three kept tokens, six experts and two
    identity ones in four groups of which two are kept, a shared expert, a layer without feed-forward."""
    moe = K.moe_mlp(experts=6, identity=2, top=3, ff=24, groups=(4, 2), shared_ff=16)
    return K.make_config([
        K.attention_spec(heads=4, kv_heads=2, dim=16, scale=0.3, rot_dims=8, size=12, keep=3, base=1000.0,
                         scaling=(3.0, 60, 4.0, 0.5), mlp=moe),
        K.distance_spec(heads=4, kv_heads=2, dim=16, vdim=24, scale=0.25, bias_max=30, rows=12, size=21, mlp=moe),
        K.attention_spec(heads=2, kv_heads=2, dim=16, scale=0.25, rot_dims=16, size=9, keep=1, base=500.0, mlp=None),
        K.distance_spec(heads=2, kv_heads=1, dim=16, vdim=8, scale=0.3, bias_max=6, rows=8, size=5, mlp=moe),
    ], width=64, vocab=96, loop=(1, 3, 2))


def config_ones():
    """What a usual model makes > 1 is 1 or absent here: one head, one key/value head, a window of one token, one kept
    token or none, no rotation in one layer, a distance table of one row and one of two, top 1 of two experts, one group,
    no identity and no shared expert, no loop, a layer that sees everything, a layer without feed-forward; sizes off the
    multiples of 8 (CUDA-core GEMMs even in 16 bits)."""
    one = K.moe_mlp(experts=2, top=1, ff=10)
    return K.make_config([
        K.attention_spec(heads=1, kv_heads=1, dim=10, scale=1.0, rot_dims=0, size=1, keep=1, mlp=one),
        K.distance_spec(heads=1, kv_heads=1, dim=6, vdim=10, scale=0.5, bias_max=3, rows=1, size=1, mlp=None),
        K.attention_spec(heads=1, kv_heads=1, dim=6, scale=0.4, rot_dims=2, size=1, keep=0, mlp=None),
        K.distance_spec(heads=3, kv_heads=1, dim=4, vdim=4, scale=0.5, bias_max=9, rows=2, size=3,
                        mlp=K.moe_mlp(experts=1, identity=1, top=1, ff=6, groups=(1, 1))),
        K.attention_spec(heads=3, kv_heads=3, dim=6, scale=0.4, rot_dims=6, mlp=one),
    ], width=36, vocab=50, eps=1e-5)


def config_wide():
    """Shapes that the tensor-core GEMMs and attention kernels tile: heads of 64 and of key 64 / value 128, grouped heads
    8 : 2 and 4 : 2; every layer inside a loop of three passes; windows that cross the cache's run length; a distance
    table that reaches its last row inside the window."""
    moe = K.moe_mlp(experts=7, identity=3, top=4, ff=64, groups=(5, 3), shared_ff=128)
    return K.make_config([
        K.attention_spec(heads=8, kv_heads=2, dim=64, scale=0.12, rot_dims=32, size=140, keep=5, base=3e5,
                         scaling=(8.0, 256, 16.0, 2.0), mlp=moe),
        K.distance_spec(heads=4, kv_heads=2, dim=64, vdim=128, scale=0.125, bias_max=90, rows=32, size=130, mlp=moe),
        K.distance_spec(heads=4, kv_heads=4, dim=64, vdim=64, scale=0.125, bias_max=50, rows=16, size=40, mlp=moe),
    ], width=256, vocab=264, loop=(0, 3, 3))


def config_far():
    """Sharp attention (weights with a gain that makes every query look at one key, wherever it is): a window of a few
    tokens beside which only the first ones stay visible, a window longer than the prompts, and no window."""
    return K.make_config([
        K.attention_spec(heads=2, kv_heads=1, dim=16, scale=0.8, rot_dims=4, size=7, keep=2, base=50.0, mlp=None),
        K.distance_spec(heads=2, kv_heads=2, dim=8, vdim=16, scale=1.2, bias_max=200, rows=20, size=500, mlp=None),
        K.attention_spec(heads=2, kv_heads=2, dim=8, scale=0.8, rot_dims=8, base=50.0,
                         mlp=K.moe_mlp(experts=3, identity=1, top=2, ff=16)),
    ], width=32, vocab=64)


def config_uneven():
    """Sizes in whole 16-byte vectors that no attention tile and few GEMM tiles fit: three query heads per key head, more
    kept tokens than the window is long, an odd number of distance rows without a window, five experts and an identity
    one in three groups, four chosen; a loop that starts at the first layer and leaves the last one out."""
    moe = K.moe_mlp(experts=5, identity=1, top=4, ff=40, groups=(3, 2), shared_ff=72)
    return K.make_config([
        K.attention_spec(heads=6, kv_heads=2, dim=24, scale=0.2, rot_dims=16, size=5, keep=20, base=3000.0, mlp=moe),
        K.distance_spec(heads=6, kv_heads=2, dim=32, vdim=80, scale=0.18, bias_max=40, rows=7, mlp=moe),
        K.attention_spec(heads=3, kv_heads=1, dim=40, scale=0.16, rot_dims=40, size=128, keep=0, base=9e3,
                         scaling=(2.0, 100, 8.0, 1.0), mlp=moe),
    ], width=192, vocab=300, loop=(0, 2, 2))


CONFIGS = {"mixed": config_mixed, "ones": config_ones, "wide": config_wide, "far": config_far, "uneven": config_uneven}
SEEDS = {"mixed": 5, "ones": 11, "wide": 8, "far": 4, "uneven": 6}
