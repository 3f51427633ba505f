"""Fudonex wiring — a hybrid decoder family behind the same ModelRunner / ForwardBatch / AttentionBackend surface as
llama.py, rimidra.py, nupovik.py, matepel.py and sugelix.py.  Every size and constant comes from the model's config
(`ModelConfig.layer_specs`, one entry per layer).

    x  = embed[token] · scale                                              fp32 residual stream
    layer:  x += m · ls1 ⊙ norm1(mixer(x));  x += m · ls2 ⊙ norm2(ff(x))   the sublayers read x itself
            norm(y) = y / rms(y) · (1 + w): it stands on the sublayer's output
    logits = cap · tanh(embed · norm(x) / cap)                             the embedding table, without its scale

mixers
  attention  grouped-query softmax attention with biased q / k / v projections, per-head RMS norms on q and k (weight
             shared by the heads) before a partial rotate-half rotation (frequencies rescaled in two regimes), values at
             unit RMS per head; a query sees a sliding window of tokens and, for the tokens before it, one mean key and
             value per complete block of `mask.pool` tokens; a learned sink per head in the softmax denominator, one
             sigmoid gate per head on the output.  With kv_from the keys and values (and their block means) are those
             another layer cached.
  mamba2     state-space duality: a short causal convolution + SiLU over x ‖ B ‖ C, S = exp(−exp(A_log) dt) S + dt B xᵀ
             per head, y = Sᵀ C + D x; SiLU(z) gate, then an RMS norm over equal parts of the row.
  delta      gated delta rule: short convolutions + SiLU on q, k, v, unit-length q and k per head, one decay per head, a
             write β (v − Sᵀ k); per-head RMS norm with a shared weight, SiLU gate.
feed-forward: W_down (silu(W_gate h) ⊙ W_up h).

Kernels: tcgen05 GEMMs (ops.linear) for 16-bit aligned shapes, the CUDA-core GEMM otherwise (float32 models, odd sizes);
every projection that reads one input is ONE GEMM; csrc/mixer_ops.cu for bias + norm + rotation + cache write of q / k /
v in one launch and for the residual update (norm of the output, layer scale, sum, and the next sublayer's operand);
csrc/attn_general*.cu over tokens and pooled blocks; csrc/head_decay.cu for the convolutions, both recurrences and the
gated group norm.  Residual stream, norms, softmax, positions and angles, convolution and matrix states, step sizes,
decays and unit vectors are fp32 in every dtype.  Single GPU.
"""
from __future__ import annotations

import math
from typing import Dict, Iterable, Optional, Tuple

import torch

from . import ops
from .attention_backend import RadixAttention
from .forward_batch_info import ForwardBatch, LogitsProcessorOutput
from .layers import LogitsProcessor
from .matepel import scaled_rotary_table
from .rimidra import RimidraDenseMLP

UNIT_EPS = 1e-6  # inside the root of the delta rule's unit vectors: fixed by the design


class _W:
    """A weight holder (same role as layers.LinearBase, without TP sharding)."""

    def __init__(self):
        self.weight: torch.Tensor = None


def _pad8(n: int) -> int:
    return -(-n // 8) * 8


_ROTARY_TABLES: Dict[tuple, Optional[torch.Tensor]] = {}


def _shared_rotary_table(rot: dict, max_positions: int, device) -> Optional[torch.Tensor]:
    """One table for all layers with the same rotation."""
    scaling = rot.get("scaling") or None
    key = (int(rot.get("dims") or 0), float(rot.get("base", 10000.0)), int(max_positions), str(device),
           tuple(sorted(scaling.items())) if scaling else None)
    if key not in _ROTARY_TABLES:
        _ROTARY_TABLES[key] = scaled_rotary_table(key[0], key[1], scaling, max_positions, device)
    return _ROTARY_TABLES[key]


class FudonexAttention:
    """q ‖ k ‖ v ‖ g are one GEMM (q ‖ g in a layer that reads another layer's cache); one launch adds the biases, norms
    and rotates q and k, norms v, and writes k and v into the cache."""

    def __init__(self, hidden: int, m: dict, layer_id: int, eps: float, max_positions: int, device):
        self.layer_id, self.eps = layer_id, eps
        self.heads, self.kv_heads = int(m["heads"]), int(m.get("kv_heads", m["heads"]))
        self.dim, self.vdim = int(m["dim"]), int(m.get("vdim", m["dim"]))
        self.kv_from = m.get("kv_from")
        rot, mask = m.get("rot") or {}, m.get("mask") or {}
        self.rot_dims = int(rot.get("dims") or 0)
        self.cos_sin = _shared_rotary_table(rot, max_positions, device)
        self.block_pool = int(mask.get("pool") or 0)
        own = self.kv_from is None
        self.sizes = [self.heads * self.dim, self.kv_heads * self.dim if own else 0,
                      self.kv_heads * self.vdim if own else 0, self.heads]
        self.attn = RadixAttention(self.heads, self.dim, float(m["scale"]), num_kv_heads=self.kv_heads, layer_id=layer_id,
                                   v_head_dim=self.vdim, sliding_window_size=int(mask.get("size") or -1), general=True,
                                   block_pool=self.block_pool)
        self.in_proj, self.o_proj, self.sink = _W(), _W(), _W()
        # fp32
        self.q_bias: torch.Tensor = None
        self.k_bias: torch.Tensor = None
        self.v_bias: torch.Tensor = None
        self.q_norm: torch.Tensor = None
        self.k_norm: torch.Tensor = None

    def cache_shape(self):
        return (self.kv_heads, self.dim, self.vdim) if self.kv_from is None else None

    def forward(self, h: torch.Tensor, forward_batch: ForwardBatch) -> torch.Tensor:
        self.attn.sinks = self.sink.weight  # fp32 [heads]
        y = ops.linear_any(h, self.in_proj.weight)
        q, k, v, g = y[:, : sum(self.sizes)].split(self.sizes, dim=-1)  # the GEMM's rows are padded to a multiple of 8
        q_rot = torch.empty((h.shape[0], self.sizes[0]), device=h.device, dtype=h.dtype)
        segments = [ops.rotary_segment(q, q_rot, self.heads, self.dim, self.rot_dims, bias=self.q_bias, norm_eps=self.eps,
                                       norm_weight=self.q_norm)]
        if self.kv_from is None:
            k_buf, v_buf = forward_batch.token_to_kv_pool.get_kv_buffer(self.layer_id)
            segments += [
                ops.rotary_segment(k, k_buf.view(k_buf.shape[0], -1), self.kv_heads, self.dim, self.rot_dims,
                                   bias=self.k_bias, to_pool=True, norm_eps=self.eps, norm_weight=self.k_norm),
                ops.rotary_segment(v, v_buf.view(v_buf.shape[0], -1), self.kv_heads, self.vdim, 0, bias=self.v_bias,
                                   to_pool=True, norm_eps=self.eps)]
        forward_batch.attn_backend.forward_rotary_segments(segments, forward_batch, self.cos_sin, h.dtype)
        o = self.attn(q_rot, None, None, forward_batch, save_kv_cache=False)
        return ops.linear_any(ops.head_gate_sigmoid(o, g, self.heads, self.vdim), self.o_proj.weight)

    __call__ = forward


class FudonexMamba2:
    """z ‖ x ‖ B ‖ C ‖ dt are one GEMM; x, B, C (contiguous in it) pass the convolution together; the recurrence runs with
    C as queries, B as keys and x as values."""

    form, q_scale, unit_eps = "ssd", 1.0, 0.0

    def __init__(self, hidden: int, m: dict, layer_id: int, eps: float):
        self.layer_id, self.eps = layer_id, eps
        self.num_heads, self.v_head_dim, self.head_dim = int(m["heads"]), int(m["vdim"]), int(m["state"])
        self.num_k_heads, self.taps, self.norm_groups = int(m["groups"]), int(m["conv"]), int(m["norm_groups"])
        self.inner, self.bc = self.num_heads * self.v_head_dim, self.num_k_heads * self.head_dim
        self.channels = self.inner + 2 * self.bc
        self.in_proj, self.conv, self.conv_bias, self.norm, self.o_proj = (_W() for _ in range(5))
        # fp32 [heads]
        self.dt_bias: torch.Tensor = None
        self.a_log: torch.Tensor = None
        self.skip: torch.Tensor = None

    def forward(self, h: torch.Tensor, forward_batch: ForwardBatch) -> torch.Tensor:
        y = ops.linear_any(h, self.in_proj.weight)
        sizes = [self.inner, self.channels, self.num_heads]
        z, xbc, dt = y[:, : sum(sizes)].split(sizes, dim=-1)
        backend = forward_batch.attn_backend
        xbc = backend.forward_short_conv(xbc, self.conv.weight, self.conv_bias.weight, self, forward_batch)
        x, b, c = xbc.split([self.inner, self.bc, self.bc], dim=-1)
        o = backend.forward_head_decay(c, b, x, dt, self, forward_batch)
        return ops.linear_any(ops.gated_group_norm(o, z, self.norm.weight, self.norm_groups, self.eps), self.o_proj.weight)

    __call__ = forward


class FudonexDelta:
    """q ‖ k ‖ v ‖ g ‖ b ‖ a are one GEMM; q, k, v pass one convolution (their taps stacked)."""

    form, unit_eps, skip = "delta", UNIT_EPS, None

    def __init__(self, hidden: int, m: dict, layer_id: int, eps: float):
        self.layer_id, self.eps = layer_id, eps
        self.num_heads, self.num_k_heads = int(m["heads"]), int(m.get("kv_heads", m["heads"]))
        self.head_dim, self.v_head_dim, self.taps = int(m["dim"]), int(m.get("vdim", m["dim"])), int(m["conv"])
        self.q_scale = self.head_dim ** -0.5
        self.qk_size, self.v_size = self.num_k_heads * self.head_dim, self.num_heads * self.v_head_dim
        self.channels = 2 * self.qk_size + self.v_size
        self.in_proj, self.conv, self.norm, self.o_proj = (_W() for _ in range(4))
        # fp32 [heads]
        self.dt_bias: torch.Tensor = None
        self.a_log: torch.Tensor = None

    def forward(self, h: torch.Tensor, forward_batch: ForwardBatch) -> torch.Tensor:
        y = ops.linear_any(h, self.in_proj.weight)
        sizes = [self.channels, self.v_size, self.num_heads, self.num_heads]
        qkv, g, b, a = y[:, : sum(sizes)].split(sizes, dim=-1)
        backend = forward_batch.attn_backend
        qkv = backend.forward_short_conv(qkv, self.conv.weight, None, self, forward_batch)
        q, k, v = qkv.split([self.qk_size, self.qk_size, self.v_size], dim=-1)
        o = backend.forward_head_decay(q, k, v, a, self, forward_batch, b=b)
        y = ops.headnorm_gate(o, g, self.num_heads, self.v_head_dim, self.eps, weight=self.norm.weight)
        return ops.linear_any(y, self.o_proj.weight)

    __call__ = forward


class FudonexDecoderLayer:
    def __init__(self, config, layer_id: int, device):
        spec = config.layer_specs[layer_id]
        H, eps, m = config.hidden_size, config.rms_norm_eps, spec["mixer"]
        self.layer_id, self.kind = layer_id, spec["type"]
        # what multiplies a sublayer's output at unit RMS before it is added: m · ls · (1 + w), fp32 [width]
        self.coef1: torch.Tensor = None
        self.coef2: torch.Tensor = None
        self.mixer = (FudonexAttention(H, m, layer_id, eps, config.max_position_embeddings, device)
                      if self.kind == "attention" else
                      (FudonexMamba2 if self.kind == "mamba2" else FudonexDelta)(H, m, layer_id, eps))
        self.mlp = RimidraDenseMLP(H, spec["mlp"], act="silu") if spec.get("mlp") is not None else None


class FudonexForCausalLM:
    def __init__(self, config, dtype=torch.bfloat16, device="cuda"):
        if config.layer_specs is None:
            raise ValueError("FudonexForCausalLM needs ModelConfig.layer_specs")
        self.config, self.dtype, self.device = config, dtype, device
        self.eps = config.rms_norm_eps
        self.embed_scale = float(config.embedding_scale)
        self.residual_mult = float(config.residual_mult)
        self.softcap = config.logit_softcap
        self.embed_tokens, self.final_norm = _W(), _W()
        self.layers = [FudonexDecoderLayer(config, i, device) for i in range(config.num_hidden_layers)]
        self.logits_processor = LogitsProcessor(config)

    def cache_shapes(self):
        """(kv shapes, matrix-state shapes, vector-state sizes, extras) per layer — what ModelRunner sizes the pools with.
        An attention layer owns (kv heads, dim, vdim) per token unless it reads another layer's; a recurrent layer owns a
        state (heads, v_dim, key dim) and the last taps − 1 inputs of its convolution per request."""
        kv, st, sh = [], [], []
        for layer in self.layers:
            m = layer.mixer
            if layer.kind == "attention":
                kv.append(m.cache_shape()), st.append(None), sh.append(None)
            else:
                kv.append(None), st.append((m.num_heads, m.v_head_dim, m.head_dim))
                sh.append((m.taps - 1) * m.channels or None)
        attn = [layer.mixer if layer.kind == "attention" else None for layer in self.layers]
        return kv, st, sh, {"kv_from": [m.kv_from if m else None for m in attn],
                            "block_sizes": [(m.block_pool or None) if m else None for m in attn]}

    @torch.no_grad()
    def forward(self, input_ids, positions, forward_batch: ForwardBatch, input_embeds=None) -> LogitsProcessorOutput:
        x = ops.embed_pair(self.embed_tokens.weight, input_ids, self.embed_scale)  # fp32, updated in place from here on
        h = ops.residual_postnorm(x, None, None, self.eps, self.dtype)
        rows = self.logits_processor.logit_rows(forward_batch)
        hook = getattr(self, "_layer_hook", None)
        last = self.layers[-1]
        for layer in self.layers:
            # the update after the model's last sublayer also norms x for the head when every row is wanted
            fin = dict(weight=self.final_norm.weight, weight_offset=1.0) if layer is last and rows is None else {}
            y = layer.mixer(h, forward_batch)
            h = ops.residual_postnorm(x, y, layer.coef1, self.eps, self.dtype, **(fin if layer.mlp is None else {}))
            if layer.mlp is not None:
                h = ops.residual_postnorm(x, layer.mlp(h), layer.coef2, self.eps, self.dtype, **fin)
            if hook is not None:  # debugging / tests: the residual stream after this layer
                hook(layer.layer_id, x.clone())
        if rows is not None and rows.numel() == 0:  # a portion whose logits nobody asked for
            return LogitsProcessorOutput(next_token_logits=torch.empty(
                (0, self.config.vocab_size), device=x.device, dtype=torch.float32))
        if rows is not None:
            h = ops.residual_postnorm(ops.embed_f32(x, rows), None, None, self.eps, self.dtype,
                                      weight=self.final_norm.weight, weight_offset=1.0)  # fp32 row gather, then the norm
        logits = ops.linear_any(h, self.embed_tokens.weight, out_f32=True)
        if self.softcap:
            ops.softcap_f32_(logits, self.softcap)
        return LogitsProcessorOutput(next_token_logits=logits)

    __call__ = forward

    # ------------------------------------------------------------------------------------------
    # parameters.  Checkpoint names: embed, final.norm, l<i>.{norm1,ls1,norm2,ls2}, l<i>.mlp.{gate,up,down}, and
    # l<i>.mix.{q,q.b,q.norm,k,k.b,k.norm,v,v.b,sink,g,o} (attention; no k / v with kv_from),
    # l<i>.mix.{in,conv,conv.b,dt_bias,A_log,D,norm,o} (mamba2),
    # l<i>.mix.{q,q.conv,k,k.conv,v,v.conv,b,a,A_log,dt_bias,norm,g,o} (delta)
    # ------------------------------------------------------------------------------------------
    def full_shapes(self) -> Dict[str, Tuple[int, ...]]:
        H = self.config.hidden_size
        shapes: Dict[str, Tuple[int, ...]] = {"embed": (self.config.vocab_size, H)}
        for layer in self.layers:
            p, m = f"l{layer.layer_id}.", layer.mixer
            q = p + "mix."
            shapes.update({p + "norm1": (H,), p + "ls1": (H,)})
            if layer.kind == "attention":
                shapes.update({q + "q": (m.heads * m.dim, H), q + "q.b": (m.heads * m.dim,), q + "q.norm": (m.dim,),
                               q + "sink": (m.heads,), q + "g": (m.heads, H), q + "o": (H, m.heads * m.vdim)})
                if m.kv_from is None:
                    shapes.update({q + "k": (m.kv_heads * m.dim, H), q + "k.b": (m.kv_heads * m.dim,),
                                   q + "k.norm": (m.dim,), q + "v": (m.kv_heads * m.vdim, H),
                                   q + "v.b": (m.kv_heads * m.vdim,)})
            else:
                nh = (m.num_heads,)
                shapes.update({q + "A_log": nh, q + "dt_bias": nh})
                if layer.kind == "mamba2":
                    shapes.update({q + "in": (m.inner + m.channels + m.num_heads, H), q + "conv": (m.channels, m.taps),
                                   q + "conv.b": (m.channels,), q + "D": nh, q + "norm": (m.inner,),
                                   q + "o": (H, m.inner)})
                else:
                    for n, rows in (("q", m.qk_size), ("k", m.qk_size), ("v", m.v_size)):
                        shapes.update({q + n: (rows, H), q + n + ".conv": (rows, m.taps)})
                    shapes.update({q + "b": (m.num_heads, H), q + "a": (m.num_heads, H), q + "norm": (m.v_head_dim,),
                                   q + "g": (m.v_size, H), q + "o": (H, m.v_size)})
            if layer.mlp is not None:
                ff = layer.mlp.ff
                shapes.update({p + "norm2": (H,), p + "ls2": (H,), p + "mlp.gate": (ff, H), p + "mlp.up": (ff, H),
                               p + "mlp.down": (H, ff)})
        shapes["final.norm"] = (H,)
        return shapes

    def load_weights(self, weights: Iterable[Tuple[str, torch.Tensor]]):
        w = {k: v for k, v in weights}
        shapes = self.full_shapes()
        missing = set(shapes) - set(w)
        if missing:
            raise KeyError(f"missing parameters: {sorted(missing)[:4]} …")
        for name, shape in shapes.items():
            if tuple(w[name].shape) != tuple(shape):
                raise ValueError(f"{name}: shape {tuple(w[name].shape)} does not match the config's {tuple(shape)}")

        def put(t):
            return t.to(self.dtype).to(self.device).contiguous()

        def put32(t):
            return t.to(torch.float32).to(self.device).contiguous()

        def rows8(names):
            t = torch.cat([w[n] for n in names], 0)
            pad = _pad8(t.shape[0]) - t.shape[0]
            return put(torch.cat([t, t.new_zeros((pad, t.shape[1]))], 0) if pad else t)

        def coefficient(norm, scale):
            return put32(self.residual_mult * w[scale].double() * (1.0 + w[norm].double()))

        self.embed_tokens.weight = put(w["embed"])
        self.final_norm.weight = put(w["final.norm"])
        for layer in self.layers:
            p, mx = f"l{layer.layer_id}.", layer.mixer
            q = p + "mix."
            layer.coef1 = coefficient(p + "norm1", p + "ls1")
            if layer.kind == "attention":
                own = mx.kv_from is None
                mx.in_proj.weight = rows8([q + n for n in (("q", "k", "v", "g") if own else ("q", "g"))])
                mx.q_bias, mx.q_norm, mx.sink.weight = put32(w[q + "q.b"]), put32(w[q + "q.norm"]), put32(w[q + "sink"])
                if own:
                    mx.k_bias, mx.k_norm, mx.v_bias = put32(w[q + "k.b"]), put32(w[q + "k.norm"]), put32(w[q + "v.b"])
            else:
                mx.dt_bias, mx.a_log, mx.norm.weight = put32(w[q + "dt_bias"]), put32(w[q + "A_log"]), put(w[q + "norm"])
                if layer.kind == "mamba2":
                    mx.in_proj.weight, mx.skip = rows8([q + "in"]), put32(w[q + "D"])
                    mx.conv.weight, mx.conv_bias.weight = put(w[q + "conv"].T), put(w[q + "conv.b"])
                else:
                    mx.in_proj.weight = rows8([q + n for n in ("q", "k", "v", "g", "b", "a")])
                    mx.conv.weight = put(torch.cat([w[q + n + ".conv"] for n in ("q", "k", "v")], 0).T)
            mx.o_proj.weight = put(w[q + "o"])
            if layer.mlp is not None:
                layer.coef2 = coefficient(p + "norm2", p + "ls2")
                layer.mlp.gate_up_proj.weight = put(torch.cat([w[p + "mlp.gate"], w[p + "mlp.up"]], 0))
                layer.mlp.down_proj.weight = put(w[p + "mlp.down"])

    def dummy_full_weights(self, seed: int = 1234) -> Dict[str, torch.Tensor]:
        """Random weights by checkpoint name: projections N(0, 1/fan_in), layer scales, skips and the per-head norm weights
        around 1, the weights stored around zero and the other vectors N(0, 0.1²), decay rates exp(A_log) around 1 and
        step sizes around 0.1, embedding rows of unit scale divided by the embedding's multiplier; rounded to bfloat16
        like a stored checkpoint; one generator per parameter."""
        out = {}
        for idx, (name, shape) in enumerate(self.full_shapes().items()):
            g = torch.Generator().manual_seed(seed + idx)
            last = name.split(".")[-1]
            if last in ("ls1", "ls2", "D") or name.endswith(("q.norm", "k.norm", "mix.norm")):
                t = 1.0 + torch.randn(shape, generator=g) * 0.1
            elif last == "dt_bias":
                t = -2.0 + torch.randn(shape, generator=g) * 0.5
            elif last == "conv":
                t = torch.randn(shape, generator=g) / math.sqrt(shape[-1])
            elif len(shape) == 1:
                t = torch.randn(shape, generator=g) * 0.1
            elif name == "embed":
                t = torch.randn(shape, generator=g) / max(self.embed_scale, 1e-6)
            else:
                t = torch.randn(shape, generator=g) / math.sqrt(shape[-1])
            out[name] = t.to(torch.bfloat16)
        return out

    def init_dummy_weights(self, seed: int = 1234):
        w = self.dummy_full_weights(seed)
        self.load_weights(w.items())
        return w
