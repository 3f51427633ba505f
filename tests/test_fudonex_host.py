"""Host side of the Fudonex family, no GPU: the config reader and its refusals, the checkpoint checks and layout of
load_weights, the pools the model asks for (a cache shared between layers, block rows behind the token rows, convolution
and transposed matrix states), the address rule of the block rows, and the oracle's own consistency (two-token form of the
delta rule, blocks, frequency rescaling)."""
import json

import pytest
import torch

from oracle import fudonex_oracle as F
from tests import fudonex_helpers as C
from tests import rimidra_helpers as H


def _folder(tmp_path, cfg, weights=None):
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    if weights is not None:
        H.write_safetensors(str(tmp_path / "model.safetensors"), weights)
    return str(tmp_path)


@pytest.mark.parametrize("name", list(C.CONFIGS))
def test_config_reader(tmp_path, name):
    from semi_pd_b200.configs import get_model_config
    cfg = C.CONFIGS[name]()
    mc = get_model_config(_folder(tmp_path, cfg))
    assert mc.model_type == "fudonex" and mc.num_hidden_layers == len(cfg["layers"])
    assert mc.hidden_size == cfg["width"] and mc.vocab_size == cfg["vocab"] and mc.rms_norm_eps == cfg["norm"]["eps"]
    assert mc.embedding_scale == cfg["embedding"]["scale"] and mc.residual_mult == cfg["residual_mult"]
    assert mc.logit_softcap == cfg.get("logit_softcap")
    assert [(s["type"], s["mixer"], s["mlp"]) for s in mc.layer_specs] == [(s["type"], s["mixer"], s["mlp"]) for s in cfg["layers"]]


def test_reader_refuses_what_it_does_not_know(tmp_path):
    from semi_pd_b200.configs import get_model_config
    good = C.config_mixed()
    for change in (lambda c: c["layers"][0].update(type="retention"),
                   lambda c: c["layers"][0]["mlp"].update(kind="moe"),
                   lambda c: c["layers"][0]["mixer"].update(heads=5),
                   lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7),
                   lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18),
                   lambda c: c["layers"][0]["mixer"]["mask"].update(pool=0),
                   lambda c: c["layers"][0]["mixer"].update(mask={"pool": 4}),
                   lambda c: c["layers"][1]["mixer"].update(groups=3),
                   lambda c: c["layers"][1]["mixer"].update(norm_groups=7),
                   lambda c: c["layers"][1]["mixer"].update(conv=0),
                   lambda c: c["layers"][2]["mixer"].update(kv_from=1),   # not an attention layer
                   lambda c: c["layers"][2]["mixer"].update(kv_from=5),   # a later layer
                   lambda c: c["layers"][4]["mixer"].update(kv_from=2),   # a layer without keys of its own
                   lambda c: c["layers"][2]["mixer"].update(vdim=16),
                   lambda c: c["layers"][3]["mixer"].update(kv_heads=3),
                   lambda c: c.update(architecture="Other")):
        cfg = json.loads(json.dumps(good))
        change(cfg)
        with pytest.raises(ValueError):
            get_model_config(_folder(tmp_path, cfg))


@pytest.mark.parametrize("name", list(C.CONFIGS))
def test_checkpoint_is_checked_and_laid_out(tmp_path, name):
    from semi_pd_b200.configs import get_model_config
    from semi_pd_b200.fudonex import FudonexForCausalLM
    cfg = C.CONFIGS[name]()
    w = C.make_weights(name, cfg)
    model = FudonexForCausalLM(get_model_config(_folder(tmp_path, cfg)), dtype=torch.float32, device="cpu")
    assert {k: tuple(v) for k, v in model.full_shapes().items()} == {k: tuple(v) for k, v in F.tensor_shapes(cfg).items()}
    model.load_weights(w.items())
    kv, st, vec, extras = model.cache_shapes()
    for i, (layer, spec) in enumerate(zip(model.layers, cfg["layers"])):
        m, mx, p = spec["mixer"], layer.mixer, f"l{i}.mix."
        mask = m.get("mask") or {}
        assert extras["kv_from"][i] == m.get("kv_from") and extras["block_sizes"][i] == mask.get("pool")
        want = cfg["residual_mult"] * w[f"l{i}.ls1"].double() * (1 + w[f"l{i}.norm1"].double())
        assert torch.allclose(layer.coef1.double(), want, rtol=1e-6)
        assert (layer.coef2 is None) == (spec["mlp"] is None)
        if spec["type"] == "attention":
            own = m.get("kv_from") is None
            assert kv[i] == ((m["kv_heads"], m["dim"], m["vdim"]) if own else None) and st[i] is None and vec[i] is None
            assert mx.in_proj.weight.shape[0] % 8 == 0
            assert torch.equal(mx.in_proj.weight[: m["heads"] * m["dim"]], w[p + "q"].float())
            first_gate = sum(mx.sizes[:3])
            assert torch.equal(mx.in_proj.weight[first_gate: first_gate + m["heads"]], w[p + "g"].float())
            assert (mx.k_bias is None) == (not own)
        else:
            dk = m["state"] if spec["type"] == "mamba2" else m["dim"]
            assert kv[i] is None and st[i] == (m["heads"], m["vdim"], dk)
            assert vec[i] == ((m["conv"] - 1) * mx.channels or None) and mx.conv.weight.shape == (m["conv"], mx.channels)
            if spec["type"] == "delta":
                conv = torch.cat([w[p + n + ".conv"] for n in "qkv"], 0).float()
                assert torch.equal(mx.conv.weight.T, conv)
    some = "l0.mix.o"
    bad = dict(w)
    del bad[some]
    with pytest.raises(KeyError):
        model.load_weights(bad.items())
    bad = dict(w)
    bad[some] = bad[some][:, :-1]
    with pytest.raises(ValueError):
        model.load_weights(bad.items())


def test_pool_shares_caches_and_appends_block_rows():
    from semi_pd_b200.memory_pool import HybridTokenToKVPool
    shapes = [(2, 8, 12), None, None, (1, 4, 4), None]
    kv_from, blocks = [None, None, 0, None, 0], [16, None, 5, None, 16]
    pool = HybridTokenToKVPool(512, 1, torch.float32, shapes, "cpu", kv_from=kv_from, block_sizes=blocks)
    runs = 4
    rows = 513 + runs * 8 + runs * 26  # blocks of 16: 8 per run of 128, of 5: at most 26
    assert pool.get_key_buffer(0).shape == (rows, 2, 8) and pool.get_value_buffer(0).shape == (rows, 2, 12)
    assert pool.get_key_buffer(2) is pool.get_key_buffer(0) and pool.get_value_buffer(4) is pool.get_value_buffer(0)
    assert pool.get_key_buffer(3).shape == (513, 1, 4) and pool.get_key_buffer(1) is None
    assert pool.get_blocks(0) == (16, 128, 513) == pool.get_blocks(4) and pool.get_blocks(2) == (5, 128, 513 + runs * 8)
    assert pool.get_blocks(3) is None
    assert [pool.writes_blocks(i) for i in range(5)] == [True, False, True, False, False]
    k, v = pool.get_kv_size_bytes()
    assert (k, v) == (4 * (rows * 16 + 513 * 4), 4 * (rows * 24 + 513 * 4))
    per = HybridTokenToKVPool.bytes_per_token(shapes, torch.float32, kv_from, blocks)
    assert per * 512 >= (k + v) - 4 * (40 + 8), "the budget covers the block rows"
    for bad_from in ([None, None, 1, None, None], [None, None, 3, None, None], [None, None, 0, 0, None]):
        with pytest.raises(ValueError):
            HybridTokenToKVPool(512, 1, torch.float32, shapes, "cpu", kv_from=bad_from)


@pytest.mark.parametrize("size", [1, 2, 5, 16, 48, 128, 200, 300])
def test_block_rows_are_distinct_whatever_the_block_size(size):
    """The address rule (run of the block's last token, offset in the run / size) gives every block of every live request
    a row of its own inside the region."""
    from semi_pd_b200.memory_pool import HybridTokenToKVPool, TokenToKVPoolAllocator
    pool = HybridTokenToKVPool(2048, 1, torch.float32, [(1, 1, 1)], "cpu", block_sizes=[size])
    alloc = TokenToKVPoolAllocator(2048, torch.float32, "cpu", pool)
    alloc.alloc_extend([3, 5], [0, 0], [700, 130])
    alloc.alloc_extend([3, 5], [700, 130], [703, 900])
    p, run, base = pool.get_blocks(0)
    per = -(-run // p)
    seen = set()
    for req in (3, 5):
        slots = alloc.req_slots(req)
        for b in range(len(slots) // p):
            s = int(slots[b * p + p - 1]) - 1
            seen.add(base + (s // run) * per + (s % run) // p)
    total = 703 // p + 900 // p
    assert len(seen) == total and (not seen or (min(seen) >= base and max(seen) < pool.get_key_buffer(0).shape[0]))


def test_oracle_two_token_form_of_the_delta_rule():
    """The pairwise form that the kernel walks a prompt with is the same function as one token after the other."""
    g = torch.Generator().manual_seed(0)
    T, dk, dv = 8, 5, 3
    q, k = F.unit_vector(torch.randn(T, 1, dk, generator=g).double()), F.unit_vector(torch.randn(T, 1, dk, generator=g).double())
    v, beta = torch.randn(T, 1, dv, generator=g).double(), torch.rand(T, 1, generator=g).double()
    w = torch.rand(T, 1, generator=g).double()
    want = F.delta_recurrence(q, k, v, beta, w)[:, 0]
    S = torch.zeros(dk, dv).double()
    for t in range(0, T, 2):
        k1, k2, q1, q2 = k[t, 0], k[t + 1, 0], q[t, 0], q[t + 1, 0]
        w1, w2, b1, b2 = w[t, 0], w[t + 1, 0], beta[t, 0], beta[t + 1, 0]
        u1 = b1 * (v[t, 0] - w1 * (S.T @ k1))
        u2 = b2 * (v[t + 1, 0] - w2 * (w1 * (S.T @ k2) + (k1 @ k2) * u1))
        o1 = w1 * (S.T @ q1) + (k1 @ q1) * u1
        o2 = w2 * (w1 * (S.T @ q2) + (k1 @ q2) * u1) + (k2 @ q2) * u2
        assert torch.allclose(o1, want[t], atol=1e-12) and torch.allclose(o2, want[t + 1], atol=1e-12)
        S = w2 * (w1 * S + torch.outer(k1, u1)) + torch.outer(k2, u2)


def test_oracle_blocks_and_window_by_hand():
    """Equal scores make the softmax an average over what a query sees: count it."""
    T, window, pool = 11, 3, 2
    q, k = torch.zeros(T, 1, 2).double(), torch.zeros(T, 1, 2).double()
    v = torch.arange(T).double().view(T, 1, 1)
    o = F.windowed_pooled_attention(q, k, v, 1.0, window=window, pool=pool)[:, 0, 0]
    for i in range(T):
        seen = [float(j) for j in range(max(0, i - window + 1), i + 1)]
        seen += [b * pool + (pool - 1) / 2 for b in range(T) if b * pool + pool - 1 <= i - window]
        assert abs(o[i].item() - sum(seen) / len(seen)) < 1e-12
    sunk = F.windowed_pooled_attention(q, k, v, 1.0, window=window, pool=pool, sinks=torch.zeros(1))[:, 0, 0]
    assert abs(sunk[10].item() - o[10].item() * 7 / 8) < 1e-12  # three tokens, four blocks, one sink


def test_frequency_rescaling_agrees_with_the_product_table():
    from semi_pd_b200.matepel import scaled_rotary_table
    for dims, base, sc in ((8, 500.0, dict(factor=4.0, original=60, fast=3.0, slow=0.5)),
                           (64, 3e4, dict(factor=8.0, original=100, fast=4.0, slow=1.0)), (24, 90.0, None)):
        f, mag = F.rotary_frequencies({"dims": dims, "base": base, "scaling": sc})
        ang = torch.arange(70, dtype=torch.float64)[:, None] * f
        want = torch.cat([ang.cos(), ang.sin()], -1) * mag
        assert torch.allclose(scaled_rotary_table(dims, base, sc, 70, "cpu").double(), want, atol=1e-6)
