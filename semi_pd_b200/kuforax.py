"""Kuforax wiring — an attention-only decoder family behind the same ModelRunner / ForwardBatch / AttentionBackend surface
as llama.py, rimidra.py, nupovik.py, matepel.py, sugelix.py and fudonex.py.  Every size and constant comes from the model's
config (`ModelConfig.layer_specs`, one entry per layer RUN) or from a tensor's shape.

    x  = embed[token]                                                    fp32 residual stream
    layer:  x += norm1b(mixer(norm1(x)));  x += norm2b(ff(norm2(x)))     norm(y) = y / rms(y) · (1 + w)
    a block of layers may be repeated back to back, re-using its tensors (every repetition keeps a cache to itself)
    logits = head · norm(x)

mixers
  attention    grouped-query softmax attention whose values are the projected keys; an RMS norm over the whole q row and
               the whole k row (all heads together) before a partial rotate-half rotation with frequencies rescaled in two
               regimes; a sliding window beside which a sequence's first tokens stay visible; one sigmoid gate per head.
  attention_2  grouped-query softmax attention without rotation; a learned bias per head and distance bucket (one bucket
               per distance up close, buckets spaced by its logarithm further away) joins the scaled scores inside a
               sliding window.
feed-forward: mixture of experts W_down gelu(W_up h); softmax scores over experts and identity experts (which hand their
input on), the top-k chosen by score + correction among the best groups of neighbours, weights = the chosen scores
renormalised; a shared expert is added for every token.

Kernels: tcgen05 GEMMs (ops.linear*, grouped form, GELU in the epilogue) for 16-bit aligned shapes, the CUDA-core GEMM
otherwise (float32 models, odd sizes); every projection that reads one input is ONE GEMM; csrc/mixer_ops.cu for norm +
rotation + cache write of q / k / v in one launch and for the residual update (norm of the sublayer's output, sum, norm of
the next sublayer's input: one launch per sublayer boundary); csrc/attn_general*.cu for both attentions.  Residual stream,
norms, softmax, routing, positions and angles are fp32 in every dtype.  Single GPU.
"""
from __future__ import annotations

import math
from typing import Dict, Iterable, List, Optional, Tuple

import torch

from . import ops
from .attention_backend import RadixAttention
from .forward_batch_info import ForwardBatch, LogitsProcessorOutput
from .fudonex import _shared_rotary_table
from .layers import LogitsProcessor

BIAS_ROWS = 32  # rows of a distance table where no checkpoint says otherwise (dummy weights)


class _W:
    """A weight holder (same role as layers.LinearBase, without TP sharding)."""

    def __init__(self):
        self.weight: torch.Tensor = None


def _pad8(n: int) -> int:
    return -(-n // 8) * 8


def distance_buckets(rows: int, far: float, length: Optional[int] = None) -> List[int]:
    """Row of a distance table of `rows` entries for the distances 0, 1, …: one row per distance below half = rows // 2,
    then half + ⌊ln(n / half) / ln(far / half) · (rows − half)⌋, at most the last row.  The list ends at `length` distances
    or where the last row is reached (every distance beyond has it too), whichever comes first."""
    half = rows // 2
    out: List[int] = [] if rows > 1 else [0]
    while (length is None or len(out) < length) and (not out or out[-1] < rows - 1):
        n = len(out)
        if n >= half and far <= half:
            raise ValueError(f"a distance table of {rows} rows cannot reach its last at distance {far}")
        # (the last term keeps a ratio that is a whole number on paper from falling below it in floating point)
        out.append(n if n < half else
                   min(rows - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half) + 1e-9)))
    return out


class KuforaxAttention:
    """q ‖ k ‖ g are one GEMM; one launch norms q and k as whole rows, rotates them, and writes k (normed and rotated) and
    the values (k as projected) into the cache."""

    def __init__(self, hidden: int, m: dict, layer_id: int, eps: float, max_positions: int, device):
        self.layer_id, self.eps = layer_id, eps
        self.heads, self.kv_heads, self.dim = int(m["heads"]), int(m.get("kv_heads", m["heads"])), int(m["dim"])
        self.vdim = self.dim  # the values are the keys
        rot, mask = m.get("rot") or {}, m.get("mask") or {}
        self.rot_dims = int(rot.get("dims") or 0)
        self.cos_sin = _shared_rotary_table(rot, max_positions, device)
        self.sizes = [self.heads * self.dim, self.kv_heads * self.dim, self.heads]
        self.attn = RadixAttention(self.heads, self.dim, float(m["scale"]), num_kv_heads=self.kv_heads, layer_id=layer_id,
                                   sliding_window_size=int(mask.get("size") or -1), general=True,
                                   keep_first=int(mask.get("keep_first") or 0))
        self.in_proj, self.o_proj = _W(), _W()
        self.q_norm: torch.Tensor = None  # fp32 [heads · dim]
        self.k_norm: torch.Tensor = None  # fp32 [kv_heads · dim]

    _TENSORS = ("in_proj", "o_proj", "q_norm", "k_norm")

    def share(self, other):
        for n in self._TENSORS:
            setattr(self, n, getattr(other, n))

    def forward(self, h: torch.Tensor, forward_batch: ForwardBatch) -> torch.Tensor:
        y = ops.linear_any(h, self.in_proj.weight)
        q, k, g = y[:, : sum(self.sizes)].split(self.sizes, dim=-1)  # the GEMM's rows are padded to a multiple of 8
        k_buf, v_buf = forward_batch.token_to_kv_pool.get_kv_buffer(self.layer_id)
        q_rot = torch.empty((h.shape[0], self.sizes[0]), device=h.device, dtype=h.dtype)
        forward_batch.attn_backend.forward_rotary_segments([
            ops.rotary_segment(q, q_rot, self.heads, self.dim, self.rot_dims, norm_eps=self.eps, norm_weight=self.q_norm,
                               norm_row=True),
            ops.rotary_segment(k, k_buf.view(k_buf.shape[0], -1), self.kv_heads, self.dim, self.rot_dims, to_pool=True,
                               norm_eps=self.eps, norm_weight=self.k_norm, norm_row=True),
            ops.rotary_segment(k, v_buf.view(v_buf.shape[0], -1), self.kv_heads, self.dim, 0, to_pool=True),
        ], forward_batch, self.cos_sin, h.dtype)
        o = self.attn(q_rot, None, None, forward_batch, save_kv_cache=False)
        return ops.linear_any(ops.head_gate_sigmoid(o, g, self.heads, self.dim), self.o_proj.weight)

    __call__ = forward


class KuforaxDistanceAttention:
    """q ‖ k ‖ v are one GEMM; the bias is a table [heads, distance] unrolled from the bucketed one when the weights are
    loaded."""

    def __init__(self, hidden: int, m: dict, layer_id: int, eps: float, max_positions: int, device):
        self.layer_id = layer_id
        self.heads, self.kv_heads = int(m["heads"]), int(m.get("kv_heads", m["heads"]))
        self.dim, self.vdim = int(m["dim"]), int(m.get("vdim", m["dim"]))
        self.bias_max = float(m["bias_max"])
        self.window = int((m.get("mask") or {}).get("size") or -1)
        self.sizes = [self.heads * self.dim, self.kv_heads * self.dim, self.kv_heads * self.vdim]
        self.attn = RadixAttention(self.heads, self.dim, float(m["scale"]), num_kv_heads=self.kv_heads, layer_id=layer_id,
                                   v_head_dim=self.vdim, sliding_window_size=self.window, general=True)
        self.in_proj, self.o_proj = _W(), _W()
        self.bias: torch.Tensor = None  # fp32 [heads, distances]

    _TENSORS = ("in_proj", "o_proj", "bias")

    def share(self, other):
        for n in self._TENSORS:
            setattr(self, n, getattr(other, n))

    def unroll(self, rel: torch.Tensor) -> torch.Tensor:
        """[rows, heads] → [heads, distances]: every distance a query can see, or up to the one whose row the rest share."""
        rows = distance_buckets(rel.shape[0], self.bias_max, self.window if self.window > 0 else None)
        return rel[torch.tensor(rows)].T

    def forward(self, h: torch.Tensor, forward_batch: ForwardBatch) -> torch.Tensor:
        self.attn.distance_bias = self.bias
        y = ops.linear_any(h, self.in_proj.weight)
        q, k, v = y[:, : sum(self.sizes)].split(self.sizes, dim=-1)
        return ops.linear_any(self.attn(q, k, v, forward_batch), self.o_proj.weight)

    __call__ = forward


class KuforaxExpert:
    """A dense feed-forward of the experts' form (the shared expert)."""

    def __init__(self, m: dict):
        self.ff = int(m["ff"])
        self.up_proj, self.down_proj = _W(), _W()

    def forward(self, h: torch.Tensor) -> torch.Tensor:
        return ops.linear_any(ops.linear_gelu_any(h, self.up_proj.weight), self.down_proj.weight)

    __call__ = forward


class KuforaxMoE:
    """The experts' up and down weights are stacked for the grouped GEMMs over expert-aligned 128-row tiles; identity
    experts own no rows: the combine reads the input itself for them, and adds the shared expert."""

    def __init__(self, hidden: int, m: dict):
        r = m["router"]
        self.hidden, self.num_experts, self.identity = hidden, int(r["experts"]), int(r.get("identity") or 0)
        self.top_k, self.ff = int(r["top"]), int(m["expert"]["ff"])
        groups = r.get("groups") or {}
        self.num_groups, self.keep_groups = int(groups.get("count") or 1), int(groups.get("keep") or 1)
        self.router, self.w_up, self.w_down = _W(), _W(), _W()  # [E + identity, hidden], [E · ff, hidden], [E · hidden, ff]
        self.correction: torch.Tensor = None  # fp32 [E + identity]
        self.shared = KuforaxExpert(m["shared"]) if m.get("shared") else None

    def forward(self, h: torch.Tensor) -> torch.Tensor:
        T, E = h.shape[0], self.num_experts
        z = ops.linear_any(h, self.router.weight, out_f32=True)  # rows padded to a multiple of 8
        ids, w = ops.moe_route_scores(z, E + self.identity, self.top_k, score_func="softmax", renormalize=True,
                                      correction=self.correction, num_groups=self.num_groups,
                                      keep_groups=self.keep_groups, group_top=1)
        row_token, inv_pos, tile_group = ops.moe_align(ids, E)
        xs = ops.moe_gather_scaled(h, row_token, inv_pos, None)
        act = ops.linear_grouped_any(xs, self.w_up.weight, tile_group, E, self.ff, gelu=True)
        y = ops.linear_grouped_any(act, self.w_down.weight, tile_group, E, self.hidden)
        shared = self.shared(h) if self.shared is not None else None
        return ops.moe_combine_gated(y, inv_pos, T, self.top_k, topk_w=w, shared=shared,
                                     identity=h if self.identity else None)

    __call__ = forward


_MIXERS = {"attention": KuforaxAttention, "attention_2": KuforaxDistanceAttention}


class KuforaxDecoderLayer:
    """One layer RUN: its own cache (layer_id), tensors of its own or of the first run of the layer."""

    def __init__(self, config, layer_id: int, device):
        spec = config.layer_specs[layer_id]
        self.layer_id, self.kind = layer_id, spec["type"]
        self.name_index = int(spec.get("layer", layer_id))  # index in the checkpoint's tensor names
        self.weights_of = spec.get("weights_of")
        self.norm1, self.norm2 = _W(), _W()  # in front of the sublayers, stored around zero
        self.post1: torch.Tensor = None      # behind them: 1 + w, fp32 [width]
        self.post2: torch.Tensor = None
        self.mixer = _MIXERS[self.kind](config.hidden_size, spec["mixer"], layer_id, config.rms_norm_eps,
                                        config.max_position_embeddings, device)
        self.mlp = KuforaxMoE(config.hidden_size, spec["mlp"]) if spec.get("mlp") is not None else None

    def share(self, other: "KuforaxDecoderLayer"):
        self.norm1, self.norm2, self.post1, self.post2 = other.norm1, other.norm2, other.post1, other.post2
        self.mixer.share(other.mixer)
        self.mlp = other.mlp


class KuforaxForCausalLM:
    def __init__(self, config, dtype=torch.bfloat16, device="cuda"):
        if config.layer_specs is None:
            raise ValueError("KuforaxForCausalLM needs ModelConfig.layer_specs")
        self.config, self.dtype, self.device = config, dtype, device
        self.eps = config.rms_norm_eps
        self.embed_tokens, self.final_norm, self.lm_head = _W(), _W(), _W()
        self.layers = [KuforaxDecoderLayer(config, i, device) for i in range(config.num_hidden_layers)]
        for layer in self.layers:
            if layer.weights_of is not None:
                layer.share(self.layers[layer.weights_of])
        self.logits_processor = LogitsProcessor(config)

    def cache_shapes(self):
        """(kv shapes, matrix-state shapes, vector-state sizes) per layer run — what ModelRunner sizes the pools with:
        every run owns (kv heads, dim, vdim) per token and no recurrent state."""
        n = len(self.layers)
        return [(layer.mixer.kv_heads, layer.mixer.dim, layer.mixer.vdim) for layer in self.layers], [None] * n, [None] * n

    @torch.no_grad()
    def forward(self, input_ids, positions, forward_batch: ForwardBatch, input_embeds=None) -> LogitsProcessorOutput:
        x = ops.embed_f32(self.embed_tokens.weight, input_ids)  # updated in place from here on
        rows = self.logits_processor.logit_rows(forward_batch)
        hook = getattr(self, "_layer_hook", None)

        def step(y, coef, norm):
            """x += y / rms(y) · coef (y None: no update), then the next sublayer's operand — one kernel."""
            return ops.residual_postnorm(x, y, coef, self.eps, self.dtype, weight=norm.weight, weight_offset=1.0)

        h = step(None, None, self.layers[0].norm1)
        for i, layer in enumerate(self.layers):
            after = self.layers[i + 1].norm1 if i + 1 < len(self.layers) else self.final_norm
            y = layer.mixer(h, forward_batch)
            h = step(y, layer.post1, layer.norm2 if layer.mlp is not None else after)
            if layer.mlp is not None:
                h = step(layer.mlp(h), layer.post2, after)
            if hook is not None:  # debugging / tests: the residual stream after this layer run
                hook(layer.layer_id, x.clone())
        if rows is not None and rows.numel() == 0:  # a portion whose logits nobody asked for
            return LogitsProcessorOutput(next_token_logits=torch.empty(
                (0, self.config.vocab_size), device=x.device, dtype=torch.float32))
        if rows is not None:
            x = ops.embed_f32(x, rows)  # fp32 row gather
            h = step(None, None, self.final_norm)
        return LogitsProcessorOutput(next_token_logits=ops.linear_any(h, self.lm_head.weight, out_f32=True))

    __call__ = forward

    # ------------------------------------------------------------------------------------------
    # parameters.  Checkpoint names: embed, head, final.norm, l<i>.{norm1,norm1b,norm2,norm2b},
    # l<i>.mix.{q,k,q.norm,k.norm,g,o} (attention), l<i>.mix.{q,k,v,rel,o} (attention_2),
    # l<i>.mlp.{router, correction, e<j>.{up,down}, shared.{up,down}}
    # ------------------------------------------------------------------------------------------
    def full_shapes(self) -> Dict[str, Tuple[int, ...]]:
        """Shapes by name; the rows of a distance table (a size only the tensor carries) are given as BIAS_ROWS."""
        cfg = self.config
        H = cfg.hidden_size
        shapes: Dict[str, Tuple[int, ...]] = {"embed": (cfg.vocab_size, H)}
        for layer in self.layers:
            if layer.weights_of is not None:
                continue
            p, m = f"l{layer.name_index}.", layer.mixer
            shapes.update({p + "norm1": (H,), p + "norm1b": (H,), p + "mix.q": (m.heads * m.dim, H),
                           p + "mix.k": (m.kv_heads * m.dim, H), p + "mix.o": (H, m.heads * m.vdim)})
            if layer.kind == "attention":
                shapes.update({p + "mix.q.norm": (m.heads * m.dim,), p + "mix.k.norm": (m.kv_heads * m.dim,),
                               p + "mix.g": (m.heads, H)})
            else:
                shapes.update({p + "mix.v": (m.kv_heads * m.vdim, H), p + "mix.rel": (BIAS_ROWS, m.heads)})
            mlp = layer.mlp
            if mlp is None:
                continue
            shapes.update({p + "norm2": (H,), p + "norm2b": (H,)})
            for e in range(mlp.num_experts):
                shapes.update({f"{p}mlp.e{e}.up": (mlp.ff, H), f"{p}mlp.e{e}.down": (H, mlp.ff)})
            n = mlp.num_experts + mlp.identity
            shapes.update({p + "mlp.router": (n, H), p + "mlp.correction": (n,)})
            if mlp.shared is not None:
                shapes.update({p + "mlp.shared.up": (mlp.shared.ff, H), p + "mlp.shared.down": (H, mlp.shared.ff)})
        shapes.update({"final.norm": (H,), "head": (cfg.vocab_size, H)})
        return shapes

    def load_weights(self, weights: Iterable[Tuple[str, torch.Tensor]]):
        w = {k: v for k, v in weights}
        shapes = self.full_shapes()
        missing = set(shapes) - set(w)
        if missing:
            raise KeyError(f"missing parameters: {sorted(missing)[:4]} …")
        for name, shape in shapes.items():
            got = tuple(w[name].shape)
            if name.endswith("mix.rel"):
                got, shape = got[1:], shape[1:]  # any number of rows
            if got != tuple(shape) or w[name].dim() != len(shapes[name]):
                raise ValueError(f"{name}: shape {tuple(w[name].shape)} does not match the config's {tuple(shapes[name])}")

        def put(t):
            return t.to(self.dtype).to(self.device).contiguous()

        def put32(t):
            return t.to(torch.float32).to(self.device).contiguous()

        def rows8(names):
            t = torch.cat([w[n] for n in names], 0)
            pad = _pad8(t.shape[0]) - t.shape[0]
            return put(torch.cat([t, t.new_zeros((pad, t.shape[1]))], 0) if pad else t)

        self.embed_tokens.weight, self.lm_head.weight = put(w["embed"]), put(w["head"])
        self.final_norm.weight = put(w["final.norm"])
        for layer in self.layers:
            if layer.weights_of is not None:
                continue
            p, mx, mlp = f"l{layer.name_index}.", layer.mixer, layer.mlp
            q = p + "mix."
            layer.norm1.weight, layer.post1 = put(w[p + "norm1"]), put32(1.0 + w[p + "norm1b"].float())
            if layer.kind == "attention":
                mx.in_proj.weight = rows8([q + "q", q + "k", q + "g"])
                mx.q_norm, mx.k_norm = put32(w[q + "q.norm"]), put32(w[q + "k.norm"])
            else:
                mx.in_proj.weight = rows8([q + "q", q + "k", q + "v"])
                mx.bias = put32(mx.unroll(w[q + "rel"].float()))
            mx.o_proj.weight = put(w[q + "o"])
            if mlp is None:
                continue
            layer.norm2.weight, layer.post2 = put(w[p + "norm2"]), put32(1.0 + w[p + "norm2b"].float())
            q = p + "mlp."
            mlp.w_up.weight = put(torch.cat([w[f"{q}e{e}.up"] for e in range(mlp.num_experts)], 0))
            mlp.w_down.weight = put(torch.cat([w[f"{q}e{e}.down"] for e in range(mlp.num_experts)], 0))
            mlp.router.weight, mlp.correction = rows8([q + "router"]), put32(w[q + "correction"])
            if mlp.shared is not None:
                mlp.shared.up_proj.weight, mlp.shared.down_proj.weight = put(w[q + "shared.up"]), put(w[q + "shared.down"])
        for layer in self.layers:  # later runs of a looped layer read the tensors just loaded
            if layer.weights_of is not None:
                layer.share(self.layers[layer.weights_of])

    def dummy_full_weights(self, seed: int = 1234) -> Dict[str, torch.Tensor]:
        """Random weights by checkpoint name: projections N(0, 1/fan_in), q / k norm weights around 1, the norms stored
        around zero and the corrections N(0, 0.1²), embedding rows and distance biases of unit scale; rounded to bfloat16
        like a stored checkpoint; one generator per parameter."""
        out = {}
        for idx, (name, shape) in enumerate(self.full_shapes().items()):
            g = torch.Generator().manual_seed(seed + idx)
            if name.endswith(("q.norm", "k.norm")):
                t = 1.0 + torch.randn(shape, generator=g) * 0.1
            elif len(shape) == 1:
                t = torch.randn(shape, generator=g) * 0.1
            elif name == "embed" or name.endswith("mix.rel"):
                t = torch.randn(shape, generator=g)
            else:
                t = torch.randn(shape, generator=g) / math.sqrt(shape[-1])
            out[name] = t.to(torch.bfloat16)
        return out

    def init_dummy_weights(self, seed: int = 1234):
        w = self.dummy_full_weights(seed)
        self.load_weights(w.items())
        return w
