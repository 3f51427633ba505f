"""Kuforax beside Llama and Rimidra with experts (the closest family: windowed softmax attention on the same general kernels,
fp32 stream, routed experts with a shared one) at equal size: whole-model prefill / decode throughput through the worker
(ScheduleBatch → TpModelWorker, decode through the captured CUDA graphs) and the per-kernel times of the mechanisms the
family adds, each beside the like kernel of the existing paths, with the fraction of the measured roofline.  Random
weights, synthetic tokens.  `bench.py --family kuforax` runs this; stand-alone:
python scripts/bench_kuforax.py [--sizes s,m] [--out FILE] [--no-models]."""
import argparse
import json
import os
import sys

import torch

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, ROOT)
sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))

import bench_rimidra as BR  # noqa: E402  (sizes, timing helpers, the two models set beside this one)

SIZES = {
    # the Rimidra / Llama shape of the same name, plus this family's own sizes: kept tokens, the distance table's reach,
    # identity experts (as many router outputs as a quarter of the experts)
    name: dict(z, keep=4, bias_max=z["window"] // 2, identity=z["experts"] // 4) for name, z in BR.SIZES.items()
}
VOCAB = BR.VOCAB


def kuforax_config(z):
    """Eight layer runs: rotary attention, two passes over (distance attention, rotary attention, rotary attention), then
    distance attention; every layer with routed experts (the chosen count counts identity experts too) and a shared one."""
    from semi_pd_b200.configs import _kuforax_config
    H, G, D = z["heads"], z["kv_heads"], z["dim"]
    mlp = {"kind": "moe", "router": {"experts": z["experts"], "identity": z["identity"], "top": z["top"],
                                     "groups": {"count": 2, "keep": 1}},
           "expert": {"ff": z["eff"]}, "shared": {"ff": z["eff"]}}
    rot = {"type": "attention", "mlp": mlp,
           "mixer": {"heads": H, "kv_heads": G, "dim": D, "vdim": D, "scale": D ** -0.5,
                     "mask": {"size": z["window"], "keep_first": z["keep"]},
                     "rot": {"dims": D // 2, "base": 1e6,
                             "scaling": {"factor": 4.0, "original": 2048, "fast": 24.0, "slow": 1.0}}}}
    dist = {"type": "attention_2", "mlp": mlp,
            "mixer": {"heads": H, "kv_heads": G, "dim": D, "vdim": D, "scale": D ** -0.5, "bias_max": z["bias_max"],
                      "mask": {"size": z["window"]}}}
    cfg = {"architecture": "Kuforax", "vocab": VOCAB, "width": z["width"], "norm": {"eps": 1e-6}, "context": 8192,
           "layers": [rot, dist, rot, rot, dist], "loop": {"start": 1, "stop": 4, "times": 2}}
    return _kuforax_config("kuforax-bench", cfg)


def kernel_table(z, flush):
    """Per-kernel time of this family's mechanisms and of the like kernels of the existing paths."""
    from semi_pd_b200 import ops
    from semi_pd_b200.kuforax import distance_buckets
    from semi_pd_b200.matepel import scaled_rotary_table
    hbm, tf, _ = BR.peaks()
    dev, bf = "cuda", torch.bfloat16
    H, G, D, Wd, Wn = z["heads"], z["kv_heads"], z["dim"], z["width"], z["window"]
    E, I, k, F = z["experts"], z["identity"], z["top"], z["eff"]
    n_req, L, B = 4, 2048, 64
    T = n_req * L
    rows = []

    def add(name, like, ms, flops=None, bytes_=None):
        r = {"kernel": name, "like": like, "ms": ms}
        if flops is not None:
            r["tflops"] = flops / ms / 1e9
            r["frac_of_peak"] = r["tflops"] / tf
            r["peak"] = "bf16 tensor (measured)"
        if bytes_ is not None:
            r["gbs"] = bytes_ / ms / 1e6
            r["frac_of_peak"] = r["gbs"] / hbm
            r["peak"] = "hbm (measured)"
        rows.append(r)

    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
    r_ = lambda *s: torch.randn(*s, device=dev, dtype=bf)
    ev = lambda fn: BR.event_ms(fn, flush=flush)
    rpi = torch.arange(n_req, device=dev, dtype=torch.int64)
    ext = dict(prefix_lens=i32([0] * n_req), extend_lens=i32([L] * n_req), extend_start_loc=i32([r * L for r in range(n_req)]),
               max_extend_len=L)
    rpd = torch.arange(B, device=dev, dtype=torch.int64)
    sl = torch.full((B,), L, dtype=torch.int64, device=dev)
    slots = T + 256
    r2t = torch.zeros(n_req + 64, L + 64, dtype=torch.int32, device=dev)
    for r in range(n_req):
        r2t[r, :L] = torch.arange(1 + r * L, 1 + (r + 1) * L, device=dev, dtype=torch.int32)
    r2d = torch.randint(1, slots, (B + 1, L + 64), device=dev, dtype=torch.int32)

    # ---- the two attentions, each beside the window alone ----------------------------------------------------------------
    kp, vp, q = r_(slots, G, D), r_(slots, G, D), r_(T, H * D)
    rel = torch.randn(32, H, device=dev)
    table = rel[torch.tensor(distance_buckets(32, z["bias_max"], Wn), device=dev)].T.contiguous()

    def attention(tag, like, keep=0, bias=None):
        seen = sum(min(i + 1, Wn) + min(keep, max(i + 1 - Wn, 0)) for i in range(L)) * n_req
        kw = dict(num_q_heads=H, num_kv_heads=G, head_dim=D, v_dim=D, sm_scale=D ** -0.5, window=Wn, keep_first=keep, dist_bias=bias)
        ms = ev(lambda: ops.attn_general(q, kp, vp, r2t, rpi, **ext, **kw))
        add(f"{tag}, prefill {n_req}x{L} ({H}/{G}x{D})", like, ms, flops=4.0 * H * D * seen)
        ms = ev(lambda: ops.attn_general(q[:B], kp, vp, r2d, rpd, seq_lens=sl, **kw))
        add(f"{tag}, decode B={B} ctx {L}", like, ms, bytes_=B * (min(L, Wn) + keep) * G * D * 2 * 2)

    attention(f"attn_general window {Wn} + {z['keep']} kept", "", keep=z["keep"])
    attention(f"attn_general window {Wn} + distance table of {table.shape[1]}", "", bias=table)
    attention(f"attn_general window {Wn}", "like: window with kept tokens / with a distance table")
    # ---- norm of the row + rotation + cache write, beside the norm per head ----------------------------------------------
    for n in (T, B):
        y = r_(n, (H + G) * D + H)
        qs, ks = y[:, : (H + G) * D].split([H * D, G * D], -1)
        q_out, kpool, vpool = torch.empty(n, H * D, device=dev, dtype=bf), r_(slots, G * D), r_(slots, G * D)
        cs = scaled_rotary_table(D, 1e6, None, L + 64, dev)
        half = scaled_rotary_table(D // 2, 1e6, None, L + 64, dev)
        pos, loc = torch.arange(n, device=dev) % L, torch.randperm(slots - 1, device=dev)[:n] + 1
        ones = lambda m: torch.ones(m, device=dev)
        seg = ops.rotary_segment
        moved = n * (H * D * 2 + G * D * 3) * 2
        segs = [seg(qs, q_out, H, D, D // 2, norm_eps=1e-6, norm_weight=ones(H * D), norm_row=True),
                seg(ks, kpool, G, D, D // 2, to_pool=True, norm_eps=1e-6, norm_weight=ones(G * D), norm_row=True),
                seg(ks, vpool, G, D, 0, to_pool=True)]
        ms = ev(lambda: ops.rotary_segments(segs, pos, half, bf, loc=loc))
        add(f"rotary_segments, norm of the row {n}x({H}+{G}+{G})x{D}", "", ms, bytes_=moved)
        like = [seg(qs, q_out, H, D, D, norm_eps=1e-6, norm_weight=ones(D)),
                seg(ks, kpool, G, D, D, to_pool=True, norm_eps=1e-6, norm_weight=ones(D)), seg(ks, vpool, G, D, 0, to_pool=True)]
        ms = ev(lambda: ops.rotary_segments(like, pos, cs, bf, loc=loc))
        add(f"rotary_segments, norm per head {n}x({H}+{G}+{G})x{D}", "like: norm of the row", ms, bytes_=moved)
    # ---- the step between sublayers, beside the step without a norm on the output ----------------------------------------
    for n in (T, B):
        x32, a, w1, coef = torch.randn(n, Wd, device=dev), r_(n, Wd), torch.zeros(Wd, device=dev, dtype=bf), torch.ones(Wd, device=dev)
        ms = ev(lambda: ops.residual_postnorm(x32, a, coef, 1e-6, bf, weight=w1, weight_offset=1.0))
        add(f"residual_postnorm, both norms {n}x{Wd}", "", ms, bytes_=n * Wd * 12)
        ms = ev(lambda: ops.residual_rmsnorm(x32, w1, 1e-6, a=a, weight_offset=1.0))
        add(f"residual_rmsnorm {n}x{Wd}", "like: both norms", ms, bytes_=n * Wd * 12)
    # ---- experts ---------------------------------------------------------------------------------------------------------
    for n in (T, B):
        zl, corr = torch.randn(n, -(-(E + I) // 8) * 8, device=dev), torch.zeros(E + I, device=dev)
        route = lambda: ops.moe_route_scores(zl, E + I, k, "softmax", renormalize=True, correction=corr, num_groups=2, keep_groups=1,
                                             group_top=1)
        ms = ev(route)
        add(f"moe_route_scores in groups {n}x{E + I}", "", ms, bytes_=n * (E + I) * 4 + n * k * 8)
        ms = ev(lambda: ops.moe_route_scores(zl, E, k, "sigmoid"))
        add(f"moe_route_scores {n}x{E}", "like: routing in groups", ms, bytes_=n * E * 4 + n * k * 8)
        ids, wts = route()
        chosen = int((ids < E).sum())
        ids2 = torch.randint(0, E, (n, k), device=dev, dtype=torch.int32)
        a = r_(n, Wd)
        up, down = r_(E * F, Wd), r_(E * Wd, F)
        for tag, like, ii, rows_used, ident in (("with identity experts", "", ids, chosen, a), ("", "like: ", ids2, n * k, None)):
            ms = ev(lambda: ops.moe_align(ii, E))
            add(f"moe_align {tag} {n}x{k}", like + "alignment" if like else "", ms, bytes_=n * k * 12)
            row_token, inv_pos, tile_group = ops.moe_align(ii, E)
            R = row_token.numel()
            y = r_(R, Wd)
            ms = ev(lambda: ops.moe_combine_gated(y, inv_pos, n, k, topk_w=wts, shared=a, identity=ident))
            add(f"moe_combine_gated {tag} {n}x{Wd}", like + "combine" if like else "", ms, bytes_=n * Wd * 2 * (k + 2))
            xs = ops.moe_gather_scaled(a, row_token, inv_pos, None)
            tiles = float((tile_group >= 0).sum()) * 128
            if not like:
                for act, note in ((True, ""), (False, "like: GELU in the epilogue")):
                    ms = ev(lambda: ops.linear_grouped_any(xs, up, tile_group, E, F, gelu=act))
                    name = "grouped GEMM" + (" + GELU" if act else "")
                    if n == T:
                        add(f"{name} {n}x{k} rows ({tiles:.0f} in tiles) {F}x{Wd}", note, ms, flops=2.0 * rows_used * F * Wd)
                    else:
                        add(f"{name} B={n} {F}x{Wd}", note, ms, bytes_=E * F * Wd * 2)
            else:
                gu = torch.cat([up, up], 0)
                ms = ev(lambda: ops.linear_grouped_any(xs, gu, tile_group, E, F, silu_mul=True))
                if n == T:
                    add(f"grouped GEMM + SiLU mul {n}x{k} rows {F}x{Wd}", "like: GELU in the epilogue", ms,
                        flops=4.0 * rows_used * F * Wd)
                else:
                    add(f"grouped GEMM + SiLU mul B={n} {F}x{Wd}", "like: GELU in the epilogue", ms, bytes_=2 * E * F * Wd * 2)
    a, su = r_(T, Wd), r_(2 * F, Wd)
    ms = ev(lambda: ops.linear_gelu_any(a, su[:F]))
    add(f"GEMM + GELU {T}x{F}x{Wd}", "", ms, flops=2.0 * T * F * Wd)
    ms = ev(lambda: ops.linear_any(a, su[:F]))
    add(f"GEMM {T}x{F}x{Wd}", "like: GELU in the epilogue", ms, flops=2.0 * T * F * Wd)
    ms = ev(lambda: ops.linear_silu_mul_any(a, su))
    add(f"GEMM + SiLU mul {T}x{F}x{Wd}", "like: GELU in the epilogue", ms, flops=4.0 * T * F * Wd)
    return rows


def run(sizes=("s", "m"), out=None, kernels=True, models=True):
    torch.cuda.set_device(0)
    flush = torch.zeros(160 << 20, dtype=torch.uint8, device="cuda")  # > L2, written between timed launches
    hbm, tf, src = BR.peaks()
    res = {"peaks": {"hbm_gbs": hbm, "bf16_tflops": tf, "source": src},
           "timing": "CUDA events, 3 warm-up launches, 160 MB written between timed launches", "sizes": {}}
    for name in sizes:
        z = SIZES[name]
        entry = {"shape": z, "models": {}}
        if models:
            for label, cfg in (("llama", BR.llama_config(z)), ("rimidra-moe", BR.rimidra_config(z, True)),
                               ("kuforax", kuforax_config(z))):
                entry["models"][label] = BR.model_throughput(cfg, n_prompts=4, prompt_len=2048, decode_bs=64, flush=flush)
                print(name, label, json.dumps(entry["models"][label]), file=sys.stderr, flush=True)
        if kernels:
            entry["kernels"] = kernel_table(z, flush)
            for r in entry["kernels"]:
                print(name, json.dumps(r), file=sys.stderr, flush=True)
        res["sizes"][name] = entry
    if out:
        with open(out, "w") as f:
            json.dump(res, f, indent=1)
    return res


if __name__ == "__main__":
    ap = argparse.ArgumentParser()
    ap.add_argument("--sizes", default="s,m")
    ap.add_argument("--out", default="")
    ap.add_argument("--no-kernels", action="store_true")
    ap.add_argument("--no-models", action="store_true")
    a = ap.parse_args()
    run(tuple(a.sizes.split(",")), a.out or None, not a.no_kernels, not a.no_models)
