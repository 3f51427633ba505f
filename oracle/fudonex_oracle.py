"""Plain float64 statement of the Fudonex design, one function per mechanism, over a whole sequence at once (no cache:
every query looks its keys, and the blocks it may see, up in the full list).  Slow on purpose; shares no code with the
package.  Weights are a dict by checkpoint name (any float dtype, read as float64), `cfg` is the parsed config.json.

Notation: x is the residual stream [T, width], u a sublayer's input (here x itself); H heads, G key/value heads, dk key
size, dv value size per head; p is a token's position in its sequence, counted from 0.
"""
import math
from typing import List, Optional

import torch

F64 = torch.float64
UNIT_EPS = 1e-6  # inside the root of the delta rule's unit vectors: fixed by the design


def f64(t):
    return torch.as_tensor(t).to(F64)


# ---- small pieces --------------------------------------------------------------------------------
def unit_rms(x, eps):
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return unit_rms(x, eps) * f64(w)


def rms_norm_around_one(x, w, eps):
    """The weight is stored as its distance from one."""
    return unit_rms(x, eps) * (1.0 + f64(w))


def unit_vector(x):
    return x / torch.sqrt(x.pow(2).sum(-1, keepdim=True) + UNIT_EPS)


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def soft_cap(z, cap):
    return cap * torch.tanh(z / cap)


def linear(x, w, b=None):
    y = x @ f64(w).T
    return y if b is None else y + f64(b)


# ---- embedding -------------------------------------------------------------------------------------
def embed(cfg, W, tokens):
    return f64(W["embed"])[torch.tensor(tokens)] * float((cfg.get("embedding") or {}).get("scale", 1.0))


# ---- rotary positions --------------------------------------------------------------------------------
def rotary_frequencies(rot):
    """→ (frequencies [dims / 2], magnitude of cos and sin).  scaling {factor, original, fast, slow}: channels that turn
    more than `fast` times within `original` positions keep their frequency, those below `slow` turns get it divided by
    the factor, with a linear ramp over the channels between."""
    dims, base = int(rot["dims"]), float(rot["base"])
    i = torch.arange(dims // 2, dtype=F64)
    f = torch.pow(torch.tensor(base, dtype=F64), -2.0 * i / dims)
    s = rot.get("scaling")
    if not s:
        return f, 1.0
    factor = float(s["factor"])

    def channel(turns):
        return dims * math.log(float(s["original"]) / (2 * math.pi * turns)) / (2 * math.log(base))

    lo = max(math.floor(channel(float(s["fast"]))), 0)
    hi = min(math.ceil(channel(float(s["slow"]))), dims - 1)
    ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
    return f / factor * ramp + f * (1.0 - ramp), 0.1 * math.log(factor) + 1.0


def rotate(x, positions, rot):
    """x [T, heads, d]; channel i of the first rot.dims turns with channel i + dims / 2, the rest pass."""
    dims = int((rot or {}).get("dims") or 0)
    if dims == 0:
        return x
    f, mag = rotary_frequencies(rot)
    ang = f64(positions)[:, None] * f[None, :]
    c, s = (ang.cos() * mag)[:, None, :], (ang.sin() * mag)[:, None, :]
    a, b = x[..., : dims // 2], x[..., dims // 2: dims]
    return torch.cat([a * c - b * s, b * c + a * s, x[..., dims:]], dim=-1)


# ---- attention over a window and pooled blocks ---------------------------------------------------------
def block_means(t, size):
    """[T, heads, d] → [T // size, heads, d]: mean of every complete run of `size` tokens."""
    n = t.shape[0] // size
    return t[: n * size].reshape(n, size, *t.shape[1:]).mean(1)


def windowed_pooled_attention(q, k, v, scale, window=None, pool=None, sinks=None):
    """q [T, H, dk], k [T, G, dk], v [T, G, dv] of one whole sequence.  Query t sees keys j with 0 <= t - j < window
    (window None: all j <= t) and, with a pool, the mean key / value of every block of `pool` tokens that ends at or
    before t - window.  sinks [H]: one more term exp(sink_h) in the denominator that carries no value."""
    T, H, _ = q.shape
    rep = H // k.shape[1]
    kk, vv = [k], [v]
    t, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = [(j <= t) if window is None else ((j <= t) & (t - j < window))]
    if pool:
        kk.append(block_means(k, pool)), vv.append(block_means(v, pool))
        last = torch.arange(T // pool)[None, :] * pool + pool - 1
        seen.append(last <= t - window)
    kh = torch.cat(kk, 0).repeat_interleave(rep, dim=1)  # head h reads group h // (H / G)
    vh = torch.cat(vv, 0).repeat_interleave(rep, dim=1)
    s = torch.einsum("thd,jhd->htj", q, kh) * scale
    s = s.masked_fill(~torch.cat(seen, 1)[None], float("-inf"))
    m = s.max(dim=-1, keepdim=True).values
    if sinks is not None:
        m = torch.maximum(m, f64(sinks)[:, None, None])
    e = torch.exp(s - m)
    den = e.sum(-1, keepdim=True)
    if sinks is not None:
        den = den + torch.exp(f64(sinks)[:, None, None] - m)
    return torch.einsum("htj,jhv->thv", e / den, vh)


def attention_mixer(u, W, p, m, positions, eps, kv=None):
    """→ (output, (keys, values) as the cache holds them).  kv: keys and values of another layer, used instead of
    projections of this layer's own."""
    T = u.shape[0]
    H, G, dk, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = linear(u, W[p + "q"], W[p + "q.b"]).view(T, H, dk)
    q = rotate(rms_norm(q, W[p + "q.norm"], eps), positions, m.get("rot"))
    if kv is None:
        k = linear(u, W[p + "k"], W[p + "k.b"]).view(T, G, dk)
        k = rotate(rms_norm(k, W[p + "k.norm"], eps), positions, m.get("rot"))
        v = unit_rms(linear(u, W[p + "v"], W[p + "v.b"]).view(T, G, dv), eps)
        kv = (k, v)
    mask = m.get("mask") or {}
    o = windowed_pooled_attention(q, kv[0], kv[1], float(m["scale"]), window=mask.get("size"), pool=mask.get("pool"),
                                  sinks=W[p + "sink"])
    o = o * torch.sigmoid(linear(u, W[p + "g"]))[..., None]  # one gate per head
    return linear(o.reshape(T, H * dv), W[p + "o"]), kv


# ---- short convolution ------------------------------------------------------------------------------------
def short_conv(x, w, b=None):
    """Causal convolution per channel and SiLU: x [T, C], w [C, taps] with the current token's weight last."""
    taps = w.shape[1]
    padded = torch.cat([x.new_zeros(taps - 1, x.shape[1]), x], 0)
    y = sum(padded[i: i + x.shape[0]] * f64(w)[:, i] for i in range(taps))
    return silu(y if b is None else y + f64(b))


# ---- recurrences with one decay per head ----------------------------------------------------------------------
def head_decay(z, a_log, dt_bias):
    """→ (step size, decay) [T, H]: dt = softplus(z + dt_bias), decay = exp(-exp(a_log) dt)."""
    dt = softplus(z + f64(dt_bias))
    return dt, torch.exp(-torch.exp(f64(a_log)) * dt)


def ssd_recurrence(x, B, C, dt, decay, D):
    """x [T, H, dv], B / C [T, groups, N]; S [N, dv] per head: S_t = decay S_(t-1) + dt B_t x_tᵀ, y_t = S_tᵀ C_t + D x_t."""
    T, H, dv = x.shape
    rep = H // B.shape[1]
    Bh, Ch = B.repeat_interleave(rep, 1), C.repeat_interleave(rep, 1)
    S = x.new_zeros(H, B.shape[2], dv)
    y = torch.empty_like(x)
    for t in range(T):
        S = decay[t][:, None, None] * S + dt[t][:, None, None] * Bh[t][:, :, None] * x[t][:, None, :]
        y[t] = torch.einsum("hnv,hn->hv", S, Ch[t]) + f64(D)[:, None] * x[t]
    return y


def delta_recurrence(q, k, v, beta, decay):
    """q / k [T, Hk, dk] (unit vectors, q scaled), v [T, H, dv]: decay the state, correct what it returns for k towards
    v, read with q after the write."""
    T, H, dv = v.shape
    rep = H // q.shape[1]
    qh, kh = q.repeat_interleave(rep, 1), k.repeat_interleave(rep, 1)
    S = v.new_zeros(H, q.shape[2], dv)
    o = torch.empty_like(v)
    for t in range(T):
        S = decay[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hkv,hk->hv", S, kh[t]))
        S = S + kh[t][:, :, None] * u[:, None, :]
        o[t] = torch.einsum("hkv,hk->hv", S, qh[t])
    return o


def gated_group_norm(y, z, w, groups, eps):
    """Gate first, then an RMS norm of every one of `groups` equal parts by itself, then a weight per channel."""
    y = y * silu(z)
    return unit_rms(y.view(y.shape[0], groups, -1), eps).reshape(y.shape) * f64(w)


def mamba2_mixer(u, W, p, m, eps):
    T = u.shape[0]
    H, dv, N, groups = int(m["heads"]), int(m["vdim"]), int(m["state"]), int(m["groups"])
    inner = H * dv
    z, xbc, dt = linear(u, W[p + "in"]).split([inner, inner + 2 * groups * N, H], dim=-1)
    x, B, C = short_conv(xbc, W[p + "conv"], W[p + "conv.b"]).split([inner, groups * N, groups * N], dim=-1)
    dt, decay = head_decay(dt, W[p + "A_log"], W[p + "dt_bias"])
    y = ssd_recurrence(x.reshape(T, H, dv), B.reshape(T, groups, N), C.reshape(T, groups, N), dt, decay, W[p + "D"])
    return linear(gated_group_norm(y.reshape(T, inner), z, W[p + "norm"], int(m["norm_groups"]), eps), W[p + "o"])


def delta_mixer(u, W, p, m, eps):
    T = u.shape[0]
    H, Hk, dk, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = short_conv(linear(u, W[p + "q"]), W[p + "q.conv"]).view(T, Hk, dk)
    k = short_conv(linear(u, W[p + "k"]), W[p + "k.conv"]).view(T, Hk, dk)
    v = short_conv(linear(u, W[p + "v"]), W[p + "v.conv"]).view(T, H, dv)
    beta = torch.sigmoid(linear(u, W[p + "b"]))
    _, decay = head_decay(linear(u, W[p + "a"]), W[p + "A_log"], W[p + "dt_bias"])
    o = delta_recurrence(unit_vector(q) * dk ** -0.5, unit_vector(k), v, beta, decay)
    o = rms_norm(o, W[p + "norm"], eps) * silu(linear(u, W[p + "g"])).view(T, H, dv)
    return linear(o.reshape(T, H * dv), W[p + "o"])


# ---- feed-forward and the whole model ---------------------------------------------------------------------------
def dense(u, W, p):
    return linear(silu(linear(u, W[p + "gate"])) * linear(u, W[p + "up"]), W[p + "down"])


def add_sublayer(x, y, W, norm, scale, mult, eps):
    """The norm and the channel scale act on the sublayer's output; the sublayer itself read the plain stream."""
    return x + mult * rms_norm_around_one(y, W[norm], eps) * f64(W[scale])


def forward(cfg, W, tokens: List[int], layers_out: Optional[list] = None):
    """→ logits [T, vocab]; layers_out collects the residual stream after every layer."""
    eps, mult = float(cfg["norm"]["eps"]), float(cfg.get("residual_mult", 1.0))
    positions = torch.arange(len(tokens))
    x = embed(cfg, W, tokens)
    kvs = {}
    for i, spec in enumerate(cfg["layers"]):
        p, m = f"l{i}.", spec["mixer"]
        if spec["type"] == "attention":
            y, kvs[i] = attention_mixer(x, W, p + "mix.", m, positions, eps, kv=kvs.get(m.get("kv_from")))
        elif spec["type"] == "mamba2":
            y = mamba2_mixer(x, W, p + "mix.", m, eps)
        else:
            y = delta_mixer(x, W, p + "mix.", m, eps)
        x = add_sublayer(x, y, W, p + "norm1", p + "ls1", mult, eps)
        if spec.get("mlp") is not None:
            x = add_sublayer(x, dense(x, W, p + "mlp."), W, p + "norm2", p + "ls2", mult, eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    z = linear(rms_norm_around_one(x, W["final.norm"], eps), W["embed"])
    cap = cfg.get("logit_softcap")
    return soft_cap(z, float(cap)) if cap else z


# ---- configurations and random weights for tests -------------------------------------------------------------------
def attention_spec(heads, kv_heads, dim, vdim, scale, window=None, pool=None, rot_dims=0, base=10000.0, scaling=None,
                   kv_from=None, ff=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if window is not None:
        m["mask"] = {"size": window} if pool is None else {"size": window, "pool": pool}
    if rot_dims:
        m["rot"] = {"base": base, "dims": rot_dims}
        if scaling:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": dense_mlp(ff)}


def mamba2_spec(heads, vdim, state, groups, conv, norm_groups, ff=None):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv,
                                        "norm_groups": norm_groups}, "mlp": dense_mlp(ff)}


def delta_spec(heads, kv_heads, dim, vdim, conv, ff=None):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv},
            "mlp": dense_mlp(ff)}


def dense_mlp(ff):
    return None if ff is None else {"kind": "dense", "ff": ff}


def make_config(layers, width, vocab, embed_scale=1.0, residual_mult=1.0, softcap=None, eps=1e-6):
    cfg = {"architecture": "Fudonex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers,
           "embedding": {"scale": embed_scale}, "residual_mult": residual_mult}
    if softcap is not None:
        cfg["logit_softcap"] = softcap
    return cfg


def tensor_shapes(cfg):
    H, shapes = cfg["width"], {"embed": (cfg["vocab"], cfg["width"])}
    for i, spec in enumerate(cfg["layers"]):
        p, m = f"l{i}.", spec["mixer"]
        for n in ("1", "2") if spec.get("mlp") is not None else ("1",):
            shapes[p + "norm" + n] = shapes[p + "ls" + n] = (H,)
        q = p + "mix."
        h, dv = m["heads"], m["vdim"]
        if spec["type"] == "attention":
            g, dk = m["kv_heads"], m["dim"]
            shapes.update({q + "q": (h * dk, H), q + "q.b": (h * dk,), q + "q.norm": (dk,), q + "sink": (h,), q + "g": (h, H)})
            if m.get("kv_from") is None:
                shapes.update({q + "k": (g * dk, H), q + "k.b": (g * dk,), q + "k.norm": (dk,), q + "v": (g * dv, H),
                               q + "v.b": (g * dv,)})
        elif spec["type"] == "mamba2":
            bc = m["groups"] * m["state"]
            shapes.update({q + "in": (2 * h * dv + 2 * bc + h, H), q + "conv": (h * dv + 2 * bc, m["conv"]),
                           q + "conv.b": (h * dv + 2 * bc,), q + "dt_bias": (h,), q + "A_log": (h,), q + "D": (h,),
                           q + "norm": (h * dv,)})
        else:
            g, dk, c = m["kv_heads"], m["dim"], m["conv"]
            for n, rows in (("q", g * dk), ("k", g * dk), ("v", h * dv)):
                shapes[q + n], shapes[q + n + ".conv"] = (rows, H), (rows, c)
            shapes.update({q + "b": (h, H), q + "a": (h, H), q + "A_log": (h,), q + "dt_bias": (h,), q + "norm": (dv,),
                           q + "g": (h * dv, H)})
        shapes[q + "o"] = (H, h * dv)
        if spec.get("mlp") is not None:
            ff = spec["mlp"]["ff"]
            shapes.update({p + "mlp.gate": (ff, H), p + "mlp.up": (ff, H), p + "mlp.down": (H, ff)})
    shapes["final.norm"] = (H,)
    return shapes


def random_weights(cfg, seed=0):
    """Values at which every mechanism matters: decays between 0.5 and 0.999, step sizes around 0.1, sinks of either
    sign, norm weights away from their neutral value; rounded to bfloat16 like a stored checkpoint."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        last = name.split(".")[-1]
        if last == "A_log":
            t = torch.rand(shape, generator=g) * 3.0 - 1.5
        elif last == "dt_bias":
            t = torch.rand(shape, generator=g) * 3.0 - 3.0
        elif last == "conv":
            t = torch.randn(shape, generator=g) * 0.6
        elif last in ("ls1", "ls2", "D"):
            t = 1.0 + torch.randn(shape, generator=g) * 0.3
        elif name.endswith(("q.norm", "k.norm", "mix.norm")):
            t = 1.0 + torch.randn(shape, generator=g) * 0.2
        elif len(shape) == 1 and "norm" in name:
            t = torch.randn(shape, generator=g) * 0.2
        elif last == "sink":
            t = torch.randn(shape, generator=g)
        elif len(shape) == 1:
            t = torch.randn(shape, generator=g) * 0.2
        elif name == "embed":
            t = torch.randn(shape, generator=g) / float(cfg["embedding"]["scale"])
        else:
            t = torch.randn(shape, generator=g) / math.sqrt(shape[-1])
        out[name] = t.to(torch.bfloat16)
    return out
