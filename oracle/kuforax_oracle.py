"""Plain float64 statement of the Kuforax design, one function per mechanism, over a whole sequence at once (no cache:
every query looks its keys up in the full list).  Slow on purpose; shares no code with the package.  Weights are a
dict by checkpoint name (any float dtype, read as float64), `cfg` is the parsed config.json.

Notation: x is the residual stream [T, width], u a sublayer's (normed) input; H query heads, G key/value heads, dk key
size, dv value size per head; t is a query's position, j a key's, both counted from 0 in their sequence.
"""
import math
from typing import Dict, List, Optional

import torch

F64 = torch.float64
WEIGHT_EPS = 1e-20  # added to the sum that the routing weights are divided by: fixed by the design


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


def gelu(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def linear(x, w):
    return x @ f64(w).T


def embed(W, tokens):
    return f64(W["embed"])[torch.tensor(tokens)]


# ---- rotary positions ------------------------------------------------------------------------------------
def rotary_frequencies(rot):
    """→ (angle per position of every channel pair, magnitude of cos and sin).  With scaling, pairs that turn often
    within `original` positions keep their frequency, pairs that turn rarely get 1 / factor of it, with a linear ramp
    over the pair index between."""
    dims, base = int(rot["dims"]), float(rot["base"])
    i = torch.arange(dims // 2, dtype=F64)
    f = torch.pow(torch.tensor(base, dtype=F64), -2.0 * i / dims)
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0

    def pair_that_turns(times):
        return dims * math.log(float(sc["original"]) / (2.0 * math.pi * times)) / (2.0 * math.log(base))

    lo = max(math.floor(pair_that_turns(float(sc["fast"]))), 0)
    hi = min(math.ceil(pair_that_turns(float(sc["slow"]))), dims - 1)
    ramp = torch.clamp((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    factor = float(sc["factor"])
    return f / factor * ramp + f * (1.0 - ramp), 0.1 * math.log(factor) + 1.0


def rotate(x, positions, rot):
    """x [T, heads, d]: channel i of the first rot.dims turns with channel i + dims / 2 by position · f_i."""
    dims = int((rot or {}).get("dims") or 0)
    if dims == 0:
        return x
    f, mag = rotary_frequencies(rot)
    ang = f64(positions)[:, None] * f[None, :]
    c, s = mag * ang.cos()[:, None, :], mag * ang.sin()[:, None, :]
    a, b = x[..., : dims // 2], x[..., dims // 2: dims]
    return torch.cat([a * c - b * s, b * c + a * s, x[..., dims:]], dim=-1)


# ---- softmax attention -----------------------------------------------------------------------------------
def sees(t, j, mask):
    """Key j for the query at t: not later, and inside the window or among the sequence's first kept tokens."""
    mask = mask or {}
    size, keep = mask.get("size"), int(mask.get("keep_first") or 0)
    return j <= t and (size is None or t - j < int(size) or j < keep)


def seen_matrix(T, mask):
    mask = mask or {}
    t, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= t
    if mask.get("size") is not None:
        seen = seen & ((t - j < int(mask["size"])) | (j < int(mask.get("keep_first") or 0)))
    return seen


def distance_bucket(n, rows, far):
    """Row of the bias table for a key n tokens back: one row per distance below rows // 2, then rows that are spaced by
    the logarithm of the distance, reaching the last one at `far`."""
    half = rows // 2
    if n < half or rows == 1:
        return min(n, rows - 1)
    at = math.log(n / half) / math.log(far / half) * (rows - half)
    return min(rows - 1, half + math.floor(at + 1e-9))  # (1e-9: a power that is an integer on paper)


def distance_bias(T, rel, far):
    """[H, T, T] of rel[bucket(t - j), h] (0 above the diagonal)."""
    rel = f64(rel)
    rows = torch.tensor([distance_bucket(n, rel.shape[0], far) for n in range(T)])
    d = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return rel[rows[d.clamp_min(0)]].permute(2, 0, 1)


def softmax_attention(q, k, v, scale, mask=None, bias=None):
    """q [T, H, dk], k [T, G, dk], v [T, G, dv] of one whole sequence; bias [H, T, T] joins the scaled scores."""
    T, H, _ = q.shape
    G = k.shape[1]
    kh, vh = k.repeat_interleave(H // G, dim=1), v.repeat_interleave(H // G, dim=1)  # head h reads group h // (H / G)
    s = torch.einsum("thd,jhd->htj", q, kh) * scale
    if bias is not None:
        s = s + bias
    s = s.masked_fill(~seen_matrix(T, mask)[None], float("-inf"))
    return torch.einsum("htj,jhv->thv", torch.softmax(s, dim=-1), vh)


# ---- the two mixers ------------------------------------------------------------------------------------
def normed_attention_mixer(u, W, p, m, positions, eps):
    """q and k normed as whole rows and rotated, values = the keys as projected, one sigmoid gate per head."""
    T = u.shape[0]
    H, G, d = int(m["heads"]), int(m["kv_heads"]), int(m["dim"])
    q, k = linear(u, W[p + "q"]), linear(u, W[p + "k"])
    v = k.view(T, G, d)
    q = rotate(rms_norm(q, W[p + "q.norm"], eps).view(T, H, d), positions, m.get("rot"))
    k = rotate(rms_norm(k, W[p + "k.norm"], eps).view(T, G, d), positions, m.get("rot"))
    o = softmax_attention(q, k, v, float(m["scale"]), m.get("mask"))
    o = o * torch.sigmoid(linear(u, W[p + "g"]))[:, :, None]
    return linear(o.reshape(T, H * d), W[p + "o"])


def distance_attention_mixer(u, W, p, m):
    """Grouped-query attention without positions but for a learned bias per head and distance bucket."""
    T = u.shape[0]
    H, G, dk, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q, k = linear(u, W[p + "q"]).view(T, H, dk), linear(u, W[p + "k"]).view(T, G, dk)
    v = linear(u, W[p + "v"]).view(T, G, dv)
    o = softmax_attention(q, k, v, float(m["scale"]), m.get("mask"), distance_bias(T, W[p + "rel"], float(m["bias_max"])))
    return linear(o.reshape(T, H * dv), W[p + "o"])


# ---- feed-forward ------------------------------------------------------------------------------------
def expert(h, W, p):
    return linear(gelu(linear(h, W[p + "up"])), W[p + "down"])


def choice_scores(z, correction, groups=None):
    """→ (scores s, choice scores): c = s + correction, minus infinity outside the groups that are kept (a group ranks
    by its largest choice score)."""
    s = torch.softmax(f64(z), dim=-1)
    c = s + f64(correction)
    if groups:
        T, n = c.shape
        per = n // int(groups["count"])
        best = c.view(T, int(groups["count"]), per).max(-1).values
        kept = torch.topk(best, int(groups["keep"]), dim=-1).indices
        ok = torch.zeros_like(best, dtype=torch.bool).scatter_(1, kept, True)
        c = c.masked_fill(~ok.repeat_interleave(per, dim=1), float("-inf"))
    return s, c


def route(z, correction, top, groups=None):
    """→ (chosen [T, top], weights [T, top])."""
    s, c = choice_scores(z, correction, groups)
    idx = torch.topk(c, top, dim=-1).indices
    w = s.gather(-1, idx)
    return idx, w / (w.sum(-1, keepdim=True) + WEIGHT_EPS)


def routing_margin(z, correction, top, groups=None):
    """How far the choice is from another one, per token: the least (c_i - c_j) / (s_i + s_j) over pairs of a chosen and a
    not chosen expert, and of the best experts of a kept and a dropped group — the relative change of scores that swaps
    them."""
    s, c = choice_scores(z, correction, groups)
    idx, _ = route(z, correction, top, groups)
    chosen = torch.zeros_like(c, dtype=torch.bool).scatter_(1, idx, True)
    open_ = torch.isfinite(c)

    def least(value, score, a, b):
        pair = (value[:, :, None] - value[:, None, :]) / (score[:, :, None] + score[:, None, :])
        return pair.masked_fill(~(a[:, :, None] & b[:, None, :]), float("inf")).flatten(1).min(1).values

    margin = least(c.masked_fill(~open_, 0.0), s, chosen, open_ & ~chosen)
    if groups and int(groups["keep"]) < int(groups["count"]):
        n = int(groups["count"])
        best, at = (s + f64(correction)).view(len(c), n, -1).max(-1)
        kept = open_.view(len(c), n, -1).any(-1)
        margin = torch.minimum(margin, least(best, s.view(len(c), n, -1).gather(-1, at[..., None])[..., 0], kept, ~kept))
    return margin


def mixture(h, W, p, mlp, margins: Optional[list] = None):
    r = mlp["router"]
    E, I, top = int(r["experts"]), int(r.get("identity") or 0), int(r["top"])
    z = linear(h, W[p + "router"])
    idx, w = route(z, W[p + "correction"], top, r.get("groups"))
    if margins is not None:
        margins.append(routing_margin(z, W[p + "correction"], top, r.get("groups")))
    y = torch.zeros_like(h)
    for e in range(E + I):
        share = (w * (idx == e)).sum(-1)  # the expert's weight per token, 0 where it was not chosen
        rows = share.nonzero().flatten()
        if len(rows):
            out = expert(h[rows], W, f"{p}e{e}.") if e < E else h[rows]  # the last outputs hand the input on
            y[rows] += share[rows, None] * out
    if mlp.get("shared"):
        y = y + expert(h, W, p + "shared.")
    return y


# ---- the model -------------------------------------------------------------------------------------------
def layer_runs(cfg):
    """Layer indices in execution order: layers [start, stop) run `times` times in a row."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return list(range(n))
    a, b = int(loop["start"]), int(loop["stop"])
    return list(range(a)) + list(range(a, b)) * int(loop["times"]) + list(range(b, n))


def forward(cfg, W, tokens, want_layers=False, margins: Optional[list] = None):
    """tokens of ONE sequence from position 0 → logits [T, vocab] (and the residual after every layer run).  margins:
    a list that receives routing_margin [T] of every feed-forward that runs."""
    eps = float(cfg["norm"]["eps"])
    positions = list(range(len(tokens)))
    x = embed(W, tokens)
    layers = []
    for i in layer_runs(cfg):
        spec, p = cfg["layers"][i], f"l{i}."
        u = rms_norm_around_one(x, W[p + "norm1"], eps)
        if spec["type"] == "attention":
            y = normed_attention_mixer(u, W, p + "mix.", spec["mixer"], positions, eps)
        else:
            y = distance_attention_mixer(u, W, p + "mix.", spec["mixer"])
        x = x + rms_norm_around_one(y, W[p + "norm1b"], eps)
        if spec.get("mlp") is not None:
            y = mixture(rms_norm_around_one(x, W[p + "norm2"], eps), W, p + "mlp.", spec["mlp"], margins)
            x = x + rms_norm_around_one(y, W[p + "norm2b"], eps)
        layers.append(x.clone())
    logits = linear(rms_norm_around_one(x, W["final.norm"], eps), W["head"])
    return (logits, torch.stack(layers)) if want_layers else logits


class Stepper:
    """Token-by-token use of the whole-sequence statement: keeps the tokens fed so far and recomputes."""

    def __init__(self, cfg, W):
        self.cfg, self.W, self.tokens = cfg, W, []

    def feed(self, tokens):
        """→ logits of the tokens just fed [len(tokens), vocab]."""
        self.tokens += list(tokens)
        return forward(self.cfg, self.W, self.tokens)[-len(tokens):]


# ---- configurations and random checkpoints for the tests ----------------------------------------------------
def moe_mlp(experts, top, ff, identity=0, groups=None, shared_ff=0):
    """groups: (count, keep) or None."""
    r = {"experts": experts, "top": top}
    if identity:
        r["identity"] = identity
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    m = {"kind": "moe", "router": r, "expert": {"ff": ff}}
    if shared_ff:
        m["shared"] = {"ff": shared_ff}
    return m


def attention_spec(heads, kv_heads, dim, scale, rot_dims, size=None, keep=0, base=10000.0, scaling=None, mlp=None):
    """scaling: (factor, original, fast, slow) or None."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale,
         "rot": {"dims": rot_dims, "base": base}}
    if scaling:
        m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    if size is not None:
        m["mask"] = {"size": size, "keep_first": keep}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def distance_spec(heads, kv_heads, dim, vdim, scale, bias_max, rows, size=None, mlp=None):
    """rows: rows of the bias table (a tensor's size, kept beside the spec for the checkpoint maker only)."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "bias_max": bias_max}
    if size is not None:
        m["mask"] = {"size": size}
    return {"type": "attention_2", "mixer": m, "mlp": mlp, "_rows": rows}


def make_config(layers: List[dict], width, vocab, loop=None, eps=1e-6):
    """loop: (start, stop, times) or None."""
    cfg = {"architecture": "Kuforax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if loop:
        cfg["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return cfg


def tensor_shapes(cfg) -> Dict[str, tuple]:
    D = cfg["width"]
    shapes = {"embed": (cfg["vocab"], D)}
    for i, spec in enumerate(cfg["layers"]):
        p, m = f"l{i}.", spec["mixer"]
        nh, g, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        shapes.update({p + "norm1": (D,), p + "norm1b": (D,), p + "mix.q": (nh * dk, D), p + "mix.k": (g * dk, D),
                       p + "mix.o": (D, nh * dv)})
        if spec["type"] == "attention":
            shapes.update({p + "mix.q.norm": (nh * dk,), p + "mix.k.norm": (g * dk,), p + "mix.g": (nh, D)})
        else:
            shapes.update({p + "mix.v": (g * dv, D), p + "mix.rel": (spec["_rows"], nh)})
        mlp = spec.get("mlp")
        if mlp is None:
            continue
        shapes.update({p + "norm2": (D,), p + "norm2b": (D,)})
        r, ff = mlp["router"], mlp["expert"]["ff"]
        for e in range(r["experts"]):
            shapes.update({f"{p}mlp.e{e}.up": (ff, D), f"{p}mlp.e{e}.down": (D, ff)})
        n = r["experts"] + r.get("identity", 0)
        shapes.update({p + "mlp.router": (n, D), p + "mlp.correction": (n,)})
        if mlp.get("shared"):
            sf = mlp["shared"]["ff"]
            shapes.update({p + "mlp.shared.up": (sf, D), p + "mlp.shared.down": (D, sf)})
    shapes.update({"final.norm": (D,), "head": (cfg["vocab"], D)})
    return shapes


def make_weights(cfg, seed=0, gain=1.0) -> Dict[str, torch.Tensor]:
    """Random checkpoint, rounded to bfloat16 like a stored one: projections N(0, gain² / fan_in) (routers twice that, so
    that choices are rarely close), embedding rows of unit scale, norms of q and k around `gain`, norms stored around
    zero N(0, 0.1²), distance biases of unit scale, corrections N(0, 0.1²) — some choice scores are negative."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        last = name.split(".")[-1]
        if name.endswith(("q.norm", "k.norm")):
            t = gain * (1.0 + 0.1 * torch.randn(shape, generator=g))
        elif len(shape) == 1:
            t = 0.1 * torch.randn(shape, generator=g)
        elif last in ("embed", "rel"):
            t = torch.randn(shape, generator=g)
        elif last == "router":
            t = 2.0 * torch.randn(shape, generator=g) / math.sqrt(shape[-1])
        else:
            t = gain * torch.randn(shape, generator=g) / math.sqrt(shape[-1])
        out[name] = t.to(torch.bfloat16)
    return out
