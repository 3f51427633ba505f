"""Fudonex beside Llama and Rimidra (the closest family: windowed sink attention and a recurrent mixer over the state pool,
fp32 stream, dense gated feed-forward) at equal size: whole-model prefill / decode throughput through the worker
(ScheduleBatch → TpModelWorker, decode through the captured CUDA graphs) and the per-kernel times of the mechanisms the
family adds, each beside the like kernel of the existing paths, with the fraction of the measured roofline.  Random
weights, synthetic tokens.  `bench.py --family fudonex` runs this; stand-alone:
python scripts/bench_fudonex.py [--sizes s,m] [--out FILE] [--no-models]."""
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
    # the Rimidra / Llama shape of the same name, plus this family's own sizes: a state-space mixer of twice the width in
    # heads of 64 with states of 128, key heads of the delta rule shared by two value heads, blocks of 32 tokens
    name: dict(z, state=128, ssd_vdim=64, ssd_heads=2 * z["width"] // 64, delta_kv=z["heads"] // 2, pool=32)
    for name, z in BR.SIZES.items()
}
VOCAB = BR.VOCAB


def fudonex_config(z):
    """Eight layers: state space, attention, delta rule, state space, attention over the first attention's cache, delta
    rule, attention, delta rule."""
    from semi_pd_b200.configs import _fudonex_config
    H, D = z["heads"], z["dim"]
    mlp = {"kind": "dense", "ff": z["ff"]}
    att = {"heads": H, "kv_heads": z["kv_heads"], "dim": D, "vdim": D, "scale": D ** -0.5,
           "mask": {"size": z["window"], "pool": z["pool"]},
           "rot": {"dims": D, "base": 1e6, "scaling": {"factor": 4.0, "original": 2048, "fast": 24.0, "slow": 1.0}}}
    ssd = {"type": "mamba2", "mlp": mlp, "mixer": {"heads": z["ssd_heads"], "vdim": z["ssd_vdim"], "state": z["state"],
                                                   "groups": 1, "conv": 4, "norm_groups": 1}}
    delta = {"type": "delta", "mlp": mlp, "mixer": {"heads": H, "kv_heads": z["delta_kv"], "dim": D, "vdim": D, "conv": 4}}
    own = {"type": "attention", "mlp": mlp, "mixer": att}
    lent = {"type": "attention", "mlp": mlp, "mixer": dict(att, kv_from=1)}
    cfg = {"architecture": "Fudonex", "vocab": VOCAB, "width": z["width"], "norm": {"eps": 1e-6},
           "embedding": {"scale": 16.0}, "residual_mult": 0.7, "logit_softcap": 40.0, "context": 8192,
           "layers": [ssd, own, delta, ssd, lent, delta, own, delta]}
    return _fudonex_config("fudonex-bench", cfg)


def kernel_table(z, flush):
    """Per-kernel time of this family's mechanisms and of the like kernels of the existing paths."""
    from semi_pd_b200 import ops
    from semi_pd_b200.matepel import scaled_rotary_table
    hbm, tf, _ = BR.peaks()
    dev, bf = "cuda", torch.bfloat16
    H, G, D, Wd = z["heads"], z["kv_heads"], z["dim"], z["width"]
    Wn, P, RUN = z["window"], z["pool"], 128
    n_req, L, B = 4, 2048, 64
    T = n_req * L
    rows = []

    def add(name, like, ms, flops=None, bytes_=None, peak_tf=None):
        r = {"kernel": name, "like": like, "ms": ms}
        if flops is not None:
            r["tflops"] = flops / ms / 1e9
            r["frac_of_peak"] = r["tflops"] / (peak_tf or tf)
            r["peak"] = "cuda-core fp32" if peak_tf else "bf16 tensor (measured)"
        if bytes_ is not None:
            r["gbs"] = bytes_ / ms / 1e6
            r["frac_of_peak"] = r["gbs"] / hbm
            r["peak"] = "hbm (measured)"
        rows.append(r)

    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
    rpi = torch.arange(n_req, device=dev, dtype=torch.int64)
    pre, ext, start = i32([0] * n_req), i32([L] * n_req), i32([r * L for r in range(n_req)])
    rpd = torch.arange(B, device=dev, dtype=torch.int64)
    sl = torch.full((B,), L, dtype=torch.int64, device=dev)
    loc = torch.ones(B, dtype=torch.int64, device=dev)
    extend = dict(prefix_lens=pre, extend_lens=ext, extend_start_loc=start)
    ev = lambda fn: BR.event_ms(fn, flush=flush)
    r_ = lambda *s: torch.randn(*s, device=dev, dtype=bf)

    # ---- the two recurrences, each beside retention at its own shape ---------------------------------------------------
    def recurrence(form, heads, kh, dk, dv, flops):
        state = torch.zeros(B + 1, heads, dv, dk, device=dev)
        q, k, v, zz, b = r_(T, kh * dk), r_(T, kh * dk), r_(T, heads * dv), r_(T, heads), r_(T, heads)
        kw = dict(num_heads=heads, num_k_heads=kh, head_dim=dk, v_dim=dv, form=form, dt_bias=torch.full((heads,), -2.0, device=dev),
                  a_log=torch.zeros(heads, device=dev), skip=torch.ones(heads, device=dev) if form == "ssd" else None)
        bb = (lambda n: b[:n]) if form == "delta" else (lambda n: None)
        shape = f"{heads}/{kh}x{dk}x{dv}"
        ms = ev(lambda: ops.head_decay_recurrence(q, k, v, zz, state, rpi, b=bb(T), **kw, **extend))
        add(f"head_decay {form} prefill {n_req}x{L} ({shape})", "", ms, flops=flops * heads * dk * dv * T, peak_tf=BR.FP32_CORE_TFLOPS)
        ms = ev(lambda: ops.head_decay_recurrence(q[:B], k[:B], v[:B], zz[:B], state, rpd, b=bb(B), seq_lens=sl, out_cache_loc=loc, **kw))
        add(f"head_decay {form} decode B={B} ({shape})", "", ms, bytes_=B * heads * dk * dv * 4 * 2)
        dec, rs = torch.full((heads,), 0.99, device=dev), torch.zeros(B + 1, heads, dk, dv, device=dev)
        rq, rk = r_(T, heads * dk), r_(T, heads * dk)
        ms = ev(lambda: ops.retention(rq, rk, v, rs, rpi, heads, dk, dv, dec, None, 0, 1.0, **extend))
        add(f"retention prefill {n_req}x{L} ({heads}x{dk}x{dv})", f"like: head_decay {form} prefill", ms,
            flops=4.0 * heads * dk * dv * T, peak_tf=BR.FP32_CORE_TFLOPS)
        ms = ev(lambda: ops.retention(rq[:B], rk[:B], v[:B], rs, rpd, heads, dk, dv, dec, None, 0, 1.0, seq_lens=sl, out_cache_loc=loc))
        add(f"retention decode B={B} ({heads}x{dk}x{dv})", f"like: head_decay {form} decode", ms, bytes_=B * heads * dk * dv * 4 * 2)

    recurrence("ssd", z["ssd_heads"], 1, z["state"], z["ssd_vdim"], 4.0)
    recurrence("delta", H, z["delta_kv"], D, D, 6.0)

    # ---- attention over a window and pooled blocks, beside the window alone ----------------------------------------------
    runs = n_req * L // RUN + 2
    slots = runs * RUN + 1
    base, region = slots, runs * -(-RUN // P)
    r2t = torch.zeros(B + 1, L + 64, dtype=torch.int32, device=dev)
    for r in range(n_req):
        r2t[r, :L] = torch.arange(1 + r * L, 1 + (r + 1) * L, device=dev, dtype=torch.int32)
    # decoding: every request over runs of its own
    druns = B * (L // RUN)
    dbase, dregion = druns * RUN + 1, druns * -(-RUN // P)
    r2d = torch.zeros(B + 1, L + 64, dtype=torch.int32, device=dev)
    order = torch.randperm(druns, generator=torch.Generator().manual_seed(0)).to(dev)
    for r in range(B):
        runs_r = order[r * (L // RUN): (r + 1) * (L // RUN)]
        r2d[r, :L] = (runs_r[:, None] * RUN + 1 + torch.arange(RUN, device=dev)[None]).reshape(-1).to(torch.int32)
    kp, vp, dkp, dvp = (r_(n, G, D) for n in (base + region, base + region, dbase + dregion, dbase + dregion))
    q, qd, sink = r_(T, H * D), r_(B, H * D), torch.zeros(H, device=dev)
    blocks_at = lambda i: max(i - Wn + 1, 0) // P
    win = sum(min(i + 1, Wn) for i in range(L)) * n_req
    pooled = sum(blocks_at(i) for i in range(L)) * n_req
    for tag, like, bl, dbl, pairs, seen in (
            ("window + blocks", "", (P, RUN, base), (P, RUN, dbase), win + pooled, min(L, Wn) + blocks_at(L - 1)),
            ("window", "like: window + blocks", None, None, win, min(L, Wn))):
        args = dict(num_q_heads=H, num_kv_heads=G, head_dim=D, v_dim=D, sm_scale=D ** -0.5, window=Wn, sinks=sink)
        ms = ev(lambda: ops.attn_general(q, kp, vp, r2t, rpi, max_extend_len=L, blocks=bl, **extend, **args))
        add(f"attn_general {tag}, prefill {n_req}x{L} ({H}/{G}x{D}, window {Wn})", like and like + " prefill", ms, flops=4.0 * H * D * pairs)
        ms = ev(lambda: ops.attn_general(qd, dkp, dvp, r2d, rpd, seq_lens=sl, blocks=dbl, **args))
        add(f"attn_general {tag}, decode B={B} ctx {L}", like and like + " decode", ms, bytes_=B * seen * 2 * G * D * 2)
    ms = ev(lambda: ops.pool_key_blocks(kp, vp, r2t, rpi, (P, RUN, base), prefix_lens=pre, extend_lens=ext, max_extend_len=L))
    add(f"pool_key_blocks {T}x{G}x{D} by {P}", "", ms, bytes_=2 * (T + T // P) * G * D * 2)
    ms = ev(lambda: ops.pool_key_blocks(dkp, dvp, r2d, rpd, (P, RUN, dbase), seq_lens=sl))
    add(f"pool_key_blocks decode B={B}, every request completes a block", "", ms, bytes_=2 * B * (P + 1) * G * D * 2)
    kk, vv, locs = r_(T, G * D), r_(T, G * D), torch.arange(1, T + 1, device=dev)
    ms = ev(lambda: ops.kv_store(kk, vv, kp, vp, locs))
    add(f"kv_store {T}x{G}x{D}", "like: pool_key_blocks", ms, bytes_=4 * T * G * D * 2)

    # ---- bias + norm + rotation + cache write ------------------------------------------------------------------------------
    sizes = [H * D, G * D, G * D]
    wide = r_(T, sum(sizes) + H)
    qs, ks, vs = wide[:, : sum(sizes)].split(sizes, -1)
    qb, kb, vb = (torch.randn(n, device=dev) for n in sizes)
    nw = torch.ones(D, device=dev)
    q_out = torch.empty(T, H * D, device=dev, dtype=bf)
    table = scaled_rotary_table(D, 1e6, None, L + 64, dev)
    pos = torch.arange(T, device=dev) % L
    moved = T * (H * D * 2 + G * D * 2 + G * D * 2) * 2
    k2, v2 = kp.view(kp.shape[0], -1), vp.view(vp.shape[0], -1)
    for tag, like, e in (("rotary_segments with norms", "", 1e-6), ("rotary_segments", "like: with norms", None)):
        w = nw if e is not None else None
        segs = [ops.rotary_segment(qs, q_out, H, D, D, bias=qb, norm_eps=e, norm_weight=w),
                ops.rotary_segment(ks, k2, G, D, D, bias=kb, to_pool=True, norm_eps=e, norm_weight=w),
                ops.rotary_segment(vs, v2, G, D, 0, bias=vb, to_pool=True, norm_eps=e)]
        ms = ev(lambda: ops.rotary_segments(segs, pos, table, bf, loc=locs))
        add(f"{tag} q/k/v {T}x({H}+{G}+{G})x{D}", like, ms, bytes_=moved)
    ms = ev(lambda: ops.head_gate_sigmoid(q, wide[:, sum(sizes):], H, D))
    add(f"head_gate_sigmoid {T}x{H}x{D}", "", ms, bytes_=T * H * D * 2 * 2)

    # ---- convolutions and norms ------------------------------------------------------------------------------------------------
    for tag, C, bias in (("x B C", z["ssd_heads"] * z["ssd_vdim"] + 2 * z["state"], True),
                         ("q k v", 2 * z["delta_kv"] * D + H * D, False)):
        taps = 4
        x, w, st = r_(T, C + 64), r_(taps, C), torch.zeros(B + 1, (taps - 1) * C, device=dev)
        cb = r_(C) if bias else None
        ms = ev(lambda: ops.short_conv(x[:, :C], w, cb, st, rpi, max_extend_len=L, **extend))
        add(f"short_conv {tag} {T}x{C}, {taps} taps", "", ms, bytes_=T * C * 4)
        ms = ev(lambda: ops.short_conv(x[:B, :C], w, cb, st, rpd, seq_lens=sl, out_cache_loc=loc))
        add(f"short_conv {tag} decode {B}x{C}", "", ms, bytes_=B * C * (4 + 2 * 4 * (taps - 1)))
    h, mu, sh = r_(T, 2 * Wd), torch.rand(1, 2 * Wd, device=dev).to(bf), torch.zeros(B + 1, 2 * Wd, device=dev)
    ms = ev(lambda: ops.token_shift_mix(h, mu, sh, rpi, max_extend_len=L, **extend))
    add(f"token_shift_mix, one mix {T}x{2 * Wd}", "like: short_conv", ms, bytes_=T * 2 * Wd * 4)
    ms = ev(lambda: ops.token_shift_mix(h[:B].contiguous(), mu, sh, rpd, seq_lens=sl, out_cache_loc=loc))
    add(f"token_shift_mix, one mix, decode {B}x{2 * Wd}", "like: short_conv decode", ms, bytes_=B * 2 * Wd * (4 + 2 * 4))
    inner = z["ssd_heads"] * z["ssd_vdim"]
    o32, gz, gw = torch.randn(T, inner, device=dev), r_(T, inner + 64), r_(inner)
    ms = ev(lambda: ops.gated_group_norm(o32, gz[:, :inner], gw, 1, 1e-6))
    add(f"gated_group_norm {T}x{inner}, 1 part", "", ms, bytes_=T * inner * (4 + 2 + 2))
    o32, gz = torch.randn(T, H * D, device=dev), r_(T, H * D + 64)
    ms = ev(lambda: ops.headnorm_gate(o32, gz[:, : H * D], H, D, 1e-6, weight=r_(D)))
    add(f"headnorm_gate {T}x{H * D}", "like: gated_group_norm", ms, bytes_=T * H * D * (4 + 2 + 2))
    x32, y, coef, w1 = torch.randn(T, Wd, device=dev), r_(T, Wd), torch.ones(Wd, device=dev), torch.ones(Wd, device=dev, dtype=bf)
    ms = ev(lambda: ops.residual_postnorm(x32, y, coef, 1e-6, bf))
    add(f"residual_postnorm {T}x{Wd}", "", ms, bytes_=T * Wd * (4 + 4 + 2 + 2))
    ms = ev(lambda: ops.residual_rmsnorm(x32, w1, 1e-6, a=y))
    add(f"residual_rmsnorm {T}x{Wd}", "like: residual_postnorm", ms, bytes_=T * Wd * (4 + 4 + 2 + 2))
    lg = torch.randn(B, VOCAB, device=dev)
    ms = ev(lambda: ops.softcap_f32_(lg, 40.0))
    add(f"softcap_f32 {B}x{VOCAB}", "", ms, bytes_=B * VOCAB * 8)
    ms = ev(lambda: ops.scale_f32_(lg, 1.0))
    add(f"scale_f32 {B}x{VOCAB}", "like: softcap_f32", ms, bytes_=B * VOCAB * 8)
    return rows


def run(sizes=("s", "m"), out=None, kernels=True, models=True):
    torch.cuda.set_device(0)
    flush = torch.zeros(160 << 20, dtype=torch.uint8, device="cuda")  # > L2, written between timed launches
    hbm, tf, src = BR.peaks()
    res = {"peaks": {"hbm_gbs": hbm, "bf16_tflops": tf, "source": src, "fp32_core_tflops": BR.FP32_CORE_TFLOPS},
           "timing": "CUDA events, 3 warm-up launches, 160 MB written between timed launches", "sizes": {}}
    for name in sizes:
        z = SIZES[name]
        entry = {"shape": z, "models": {}}
        for label, cfg in ((("llama", BR.llama_config(z)), ("rimidra-dense", BR.rimidra_config(z, False)),
                            ("fudonex", fudonex_config(z))) if models else ()):
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
