"""Host side of the Kuforax family, no GPU: the config reader with its loop expansion and refusals, the checkpoint checks and
layout of load_weights (distance tables with any number of rows, constants of looped runs), the distance buckets, the pools
the model asks for, and the oracle's own consistency (visibility, group choice, a sequence fed token by token)."""
import json
import math

import pytest
import torch

from oracle import kuforax_oracle as K
from tests import kuforax_helpers as C
from tests import rimidra_helpers as H


def _folder(tmp_path, cfg):
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    return str(tmp_path)


@pytest.mark.parametrize("name", list(C.CONFIGS))
def test_config_reader_lists_the_layer_runs(tmp_path, name):
    from semi_pd_b200.configs import get_model_config
    from semi_pd_b200.registry import get_model_class
    cfg = C.CONFIGS[name]()
    mc = get_model_config(_folder(tmp_path, cfg))
    runs = K.layer_runs(cfg)
    assert mc.model_type == "kuforax" and mc.num_hidden_layers == len(runs)
    assert get_model_class(mc.model_type).__name__ == "KuforaxForCausalLM"
    assert mc.hidden_size == cfg["width"] and mc.vocab_size == cfg["vocab"] and mc.rms_norm_eps == cfg["norm"]["eps"]
    assert [s["layer"] for s in mc.layer_specs] == runs
    first = {}
    for r, s in enumerate(mc.layer_specs):
        assert s["weights_of"] == first.get(s["layer"]) and s["type"] == cfg["layers"][s["layer"]]["type"]
        assert s["mixer"] == cfg["layers"][s["layer"]]["mixer"]
        first.setdefault(s["layer"], r)


def test_reader_refuses_what_it_does_not_know(tmp_path):
    from semi_pd_b200.configs import get_model_config
    good = C.config_mixed()
    get_model_config(_folder(tmp_path, good))
    for change in (lambda c: c["layers"][0].update(type="latent_attention"),
                   lambda c: c["layers"][0]["mlp"].update(kind="dense"),
                   lambda c: c["layers"][0]["mixer"].update(kv_heads=3),
                   lambda c: c["layers"][0]["mixer"].update(vdim=8),
                   lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7),
                   lambda c: c["layers"][0]["mixer"]["rot"].update(dims=32),
                   lambda c: c["layers"][0]["mixer"]["mask"].update(size=0),
                   lambda c: c["layers"][0]["mixer"]["mask"].update(keep_first=-1),
                   lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=3),
                   lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=5),
                   lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=1),
                   lambda c: c["loop"].update(stop=9),
                   lambda c: c["loop"].update(times=0),
                   lambda c: c.update(architecture="Other")):
        cfg = json.loads(json.dumps(good))
        change(cfg)
        with pytest.raises(ValueError):
            get_model_config(_folder(tmp_path, cfg))


@pytest.mark.parametrize("rows,far", [(32, 128), (32, 100), (8, 6), (7, 50), (2, 9), (1, 5), (20, 160), (10, 160)])
def test_distance_buckets(rows, far):
    from semi_pd_b200.kuforax import distance_buckets
    b = distance_buckets(rows, far)
    half = rows // 2
    assert b == [K.distance_bucket(n, rows, far) for n in range(len(b))]
    assert b[:half] == list(range(half)), "one row per distance up close"
    assert b[-1] == rows - 1 and all(x <= y for x, y in zip(b, b[1:])), "the list ends at the last row"
    assert all(K.distance_bucket(n, rows, far) == rows - 1 for n in range(len(b) - 1, 3 * far))
    assert len(b) <= far + 1
    for n in (1, 3, far // 2):
        assert distance_buckets(rows, far, n) == b[:n], "no longer than the window asks for"
    # distance `far` is the last row; rows in between follow the logarithm (integer form of the same rule)
    for n in range(half, len(b)):
        if rows > 2:
            k = max(k for k in range(rows - half + 1) if far ** k * half ** (rows - half) <= n ** (rows - half) * half ** k)
            assert b[n] == min(rows - 1, half + k)


def test_distance_buckets_that_never_reach_their_last_row():
    from semi_pd_b200.kuforax import distance_buckets
    assert distance_buckets(16, 5, 8) == list(range(8)), "the logarithmic part is not needed"
    with pytest.raises(ValueError):
        distance_buckets(16, 5, 9)


@pytest.mark.parametrize("name", list(C.CONFIGS))
def test_checkpoint_is_checked_and_laid_out(tmp_path, name):
    from semi_pd_b200.configs import get_model_config
    from semi_pd_b200.kuforax import KuforaxForCausalLM
    cfg = C.CONFIGS[name]()
    w = K.make_weights(cfg, seed=1)
    model = KuforaxForCausalLM(get_model_config(_folder(tmp_path, cfg)), dtype=torch.float32, device="cpu")
    assert set(model.full_shapes()) == set(K.tensor_shapes(cfg))
    model.load_weights(w.items())
    kv, st, vec = model.cache_shapes()
    assert all(s is None for s in st) and all(s is None for s in vec)
    for layer, shape in zip(model.layers, kv):
        m, mx, p = cfg["layers"][layer.name_index]["mixer"], layer.mixer, f"l{layer.name_index}."
        assert shape == (m["kv_heads"], m["dim"], m["vdim"])
        nq, nk = m["heads"] * m["dim"], m["kv_heads"] * m["dim"]
        assert torch.equal(mx.in_proj.weight[:nq], w[p + "mix.q"].float())
        assert torch.equal(mx.in_proj.weight[nq:nq + nk], w[p + "mix.k"].float())
        assert mx.in_proj.weight.shape[0] % 8 == 0
        assert torch.equal(layer.post1, 1.0 + w[p + "norm1b"].float())
        if layer.kind == "attention":
            assert mx.attn.keep_first == ((m.get("mask") or {}).get("keep_first", 0))
            assert torch.equal(mx.in_proj.weight[nq + nk:nq + nk + m["heads"]], w[p + "mix.g"].float())
        else:
            rel = w[p + "mix.rel"].float()
            size = (m.get("mask") or {}).get("size")
            for d in range(min(size or 400, 400)):
                want = rel[K.distance_bucket(d, rel.shape[0], m["bias_max"])]
                assert torch.equal(mx.bias[:, min(d, mx.bias.shape[1] - 1)], want), d
        if layer.mlp is not None:
            r = cfg["layers"][layer.name_index]["mlp"]["router"]
            n = r["experts"] + r.get("identity", 0)
            assert torch.equal(layer.mlp.router.weight[:n], w[p + "mlp.router"].float())
            assert torch.equal(layer.mlp.correction, w[p + "mlp.correction"].float())
        if layer.weights_of is not None:  # a later run of a looped layer reads the first run's tensors and constants
            src = model.layers[layer.weights_of]
            assert layer.norm1 is src.norm1 and layer.post1 is src.post1 and layer.mlp is src.mlp
            assert mx.in_proj is src.mixer.in_proj and mx.attn is not src.mixer.attn
            for n in ("bias", "q_norm", "k_norm"):
                assert getattr(mx, n, None) is getattr(src.mixer, n, None)
    some = next(iter(k for k in w if k.endswith("mix.o")))
    for change in (lambda b: b.pop(some), lambda b: b.update({some: b[some][:, :-1]}),
                   lambda b: b.update({k: v[:, :-1] for k, v in b.items() if k.endswith("rel")} or {some: b[some][:-1]})):
        bad = dict(w)
        change(bad)
        with pytest.raises((KeyError, ValueError)):
            model.load_weights(bad.items())


def test_dummy_weights_load(tmp_path):
    from semi_pd_b200.configs import get_model_config
    from semi_pd_b200.kuforax import BIAS_ROWS, KuforaxForCausalLM
    model = KuforaxForCausalLM(get_model_config(_folder(tmp_path, C.config_uneven())), dtype=torch.bfloat16, device="cpu")
    w = model.init_dummy_weights(7)
    assert w["l1.mix.rel"].shape == (BIAS_ROWS, 6) and model.layers[1].mixer.bias.dtype == torch.float32
    again = model.dummy_full_weights(7)
    assert all(torch.equal(w[k], again[k]) for k in w)


def test_pools_hold_a_cache_per_layer_run(tmp_path):
    from semi_pd_b200.configs import get_model_config
    from semi_pd_b200.kuforax import KuforaxForCausalLM
    from semi_pd_b200.memory_pool import HybridTokenToKVPool
    cfg = C.config_mixed()
    model = KuforaxForCausalLM(get_model_config(_folder(tmp_path, cfg)), dtype=torch.bfloat16, device="cpu")
    kv, _, _ = model.cache_shapes()
    pool = HybridTokenToKVPool(128, 1, torch.bfloat16, kv, "cpu")
    assert pool.layer_num == len(K.layer_runs(cfg)) == 6
    assert len({t.data_ptr() for t in pool.k_buffer} | {t.data_ptr() for t in pool.v_buffer}) == 12
    assert HybridTokenToKVPool.bytes_per_token(kv, torch.bfloat16) == 2 * sum(g * (dk + dv) for g, dk, dv in kv)


def test_oracle_visibility_and_buckets():
    mask = {"size": 4, "keep_first": 2}
    seen = K.seen_matrix(9, mask)
    for t in range(9):
        assert [j for j in range(9) if seen[t, j]] == [j for j in range(9) if K.sees(t, j, mask)]
    assert [j for j in range(9) if seen[8, j]] == [0, 1, 5, 6, 7, 8]
    assert [j for j in range(9) if K.seen_matrix(9, {"size": 3})[8, j]] == [6, 7, 8]
    bias = K.distance_bias(6, torch.arange(8.0).view(4, 2), 5)
    assert bias.shape == (2, 6, 6)
    assert bias[1, 5, 5 - 1] == 3.0 and bias[0, 4, 4] == 0.0
    assert K.distance_bucket(4, 4, 5) == 2 + math.floor(math.log(2) / math.log(2.5) * 2)


def test_oracle_groups_by_largest_choice_score():
    s = torch.tensor([[0.40, 0.01, 0.25, 0.24, 0.05, 0.05]], dtype=torch.float64)
    idx, w = K.route(s.log(), torch.zeros(6), 2, {"count": 3, "keep": 1})
    assert set(idx[0].tolist()) == {0, 1} and float(w.sum()) == pytest.approx(1.0)
    idx, _ = K.route(s.log(), torch.tensor([-0.5, -0.3, -9.0, -9.0, -9.0, -9.0]), 2, {"count": 3, "keep": 1})
    assert set(idx[0].tolist()) == {0, 1}


def test_oracle_identity_experts_hand_their_input_on():
    cfg = K.make_config([K.attention_spec(1, 1, 4, 1.0, 0, 3, mlp=K.moe_mlp(experts=1, identity=2, top=2, ff=4))], 8, 10)
    W = K.make_weights(cfg, seed=0)
    W["l0.mlp.correction"][1:] = 5.0
    h = torch.randn(6, 8, dtype=torch.float64)
    assert torch.allclose(K.mixture(h, W, "l0.mlp.", cfg["layers"][0]["mlp"]), h, rtol=1e-12, atol=1e-12)


@pytest.mark.parametrize("name", ["ones", "mixed"])
def test_oracle_token_by_token_equals_whole(name):
    cfg = C.CONFIGS[name]()
    W = K.make_weights(cfg, seed=2)
    toks = H.prompt(17, cfg["vocab"], 1)
    whole = K.forward(cfg, W, toks)
    st = K.Stepper(cfg, W)
    rows = [st.feed(toks[:5])] + [st.feed([t]) for t in toks[5:]]
    assert torch.allclose(torch.cat(rows), whole, rtol=1e-9, atol=1e-11)
