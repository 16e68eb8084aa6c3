"""Gated attention: causal grouped-query softmax attention over the paged cache with keys and values of different sizes
and a set of options that a model description switches on one by one (GatedAttentionSpec).

With h the mixer's input, per token at position p:
    q = Wq h, k = Wk h, v = Wv h, g = Wg h                      (one product against [Wq; Wk; Wv; Wg], float32 sums)
    q_a <- rot_p(rmsnorm(q_a) * wq),  k_b <- rot_p(rmsnorm(k_b) * wk)   per head, one norm weight for all heads
    v <- (1 - m) v + m v_first                                  (value mixing; the mixed v is what the cache holds)
    score_a(i, j) = (q_a(i) . k_b(j)) * scale,  b = a // (H / G),  j <= i in the same chunk (and inside the window)
    p_a(i, j) = exp(score) / (sum_j exp(score) + exp(sink_a))   the sink only enlarges the denominator
    out = Wo ((heads' results side by side) * sigmoid(g))       g: a gate a number of the result, or (gate_per_head) one a head
With q_bias, k_bias and v_bias the projections have biases, with o_bias the output projection; rot_pairs "neighbours" turns the numbers 2i and 2i + 1 of a
head together instead of i and i + dims / 2; with unit_rms every query and key head is divided by its root mean square behind the
rotation (no weight); with keys_as_values there is no Wv: v = k as the projection gives it, before norms and rotation.
With taps > 0, q, k and v go through a causal convolution over their request's last `taps` tokens a channel, right behind the projection
(the last taps - 1 projected rows are state); with q_temperature the queries are multiplied by a number that grows with the position;
sink_score puts one constant in place of the sinks a head. With norm_scope "projection" the two norms are over all of q and all of k at once (weights of the projections' sizes). A layer
without keys and values of its own (own_kv False) forms queries only and reads the cache of the run its LayerRun names.
Norms, rotation, scores, softmax and the gate are float32 in both engine precisions. v_first are the values that the
first layer with value mixing computed for the same tokens in the same step: that layer leaves them in the step
context (`ctx.shared`), the later ones read them there.
"""
from __future__ import annotations

from typing import List, Optional

import numpy as np
import torch

from .attention import add_into_stream_or_partials
from .base import KVNeed, LayerCache, Mixer, NormalizedRows, StateNeed
from .registry import build_part, part_class, register_part
from .spec import GatedAttentionSpec, QueryTemperatureSpec, TensorNeed

V_FIRST = "gated_attention.v_first"  # key of ctx.shared
CONV = "gated_attention.conv"        # the state's name


def query_temperatures(spec: QueryTemperatureSpec) -> np.ndarray:
    """What the query at every position is multiplied with, float64 rounded to float32."""
    steps = np.floor((np.arange(spec.max_positions, dtype=np.float64) + 1.0) / float(spec.every))
    return (1.0 + float(spec.coef) * np.log(steps + 1.0)).astype(np.float32)


class GatedAttention(Mixer):
    def __init__(self, spec: GatedAttentionSpec, env):
        super().__init__(spec, env)
        for name in ("num_heads", "num_kv_heads", "head_dim", "value_dim"):
            if getattr(spec, name) <= 0:
                raise ValueError(f"gated attention: {name} must be >= 1")
        if spec.num_heads % spec.num_kv_heads:
            raise ValueError(f"gated attention: {spec.num_heads} heads cannot share {spec.num_kv_heads} key/value heads")
        if spec.window < 0 or spec.chunk < 0:
            raise ValueError("gated attention: window and chunk must be >= 0")
        if spec.norm_scope not in ("head", "projection"):
            raise ValueError("gated attention: norm_scope is 'head' or 'projection'")
        if not spec.own_kv and (spec.value_mix is not None or spec.k_norm):
            raise ValueError("gated attention: a layer that borrows keys and values has no key norm and mixes no values")
        if spec.value_mix not in (None, "first", "mix") or (spec.value_mix == "mix" and not spec.value_mix_weight):
            raise ValueError("gated attention: value_mix is None, 'first' or 'mix' (with the name of its weight)")
        if spec.rot_pairs not in ("half", "neighbours"):
            raise ValueError("gated attention: rot_pairs is 'half' or 'neighbours'")
        if spec.unit_rms and (spec.q_norm or spec.k_norm):
            raise ValueError("gated attention: unit_rms takes the place of the norms before the rotation")
        if spec.keys_as_values and (spec.value_dim != spec.head_dim or spec.value_mix is not None or not spec.own_kv):
            raise ValueError("gated attention: keys_as_values needs values of the keys' size, keys of the layer's own and no value mixing")
        # what the row form of the query/key/value preparation does (ops.qkv_prep): it mixes no values, has no unit_rms and no keys as values
        self.row_form = bool(spec.taps or spec.v_bias or spec.q_temperature is not None or
                             (spec.norm_scope == "projection" and (spec.q_bias or spec.k_bias or spec.rot_pairs != "half")))
        if (self.row_form or spec.norm_scope == "projection") and (spec.unit_rms or spec.keys_as_values):
            raise ValueError("gated attention: unit_rms and keys_as_values go with norms a head, without convolutions, value biases and query temperatures")
        if self.row_form and spec.value_mix is not None:
            raise ValueError("gated attention: convolutions, value biases and query temperatures go without value mixing")
        if spec.taps < 0 or (spec.taps > 0 and not (spec.own_kv and spec.q_conv and spec.k_conv and spec.v_conv)):
            raise ValueError("gated attention: a convolution needs its three weights, and keys and values of the layer's own")
        if spec.sink and spec.sink_score is not None:
            raise ValueError("gated attention: sinks are a tensor or one constant")
        if spec.q_temperature is not None and not (spec.q_temperature.every > 0 and spec.q_temperature.max_positions > 0):
            raise ValueError("gated attention: a query temperature needs a positive step and a position limit")
        self.position = build_part("position", spec.position, env)
        tables = self.position.rotation_tables()
        if tables is None:
            raise ValueError("gated attention needs a position encoding with rotation tables")
        self.cos, self.sin = tables
        if self.cos is not None and 2 * self.cos.shape[1] > spec.head_dim:
            raise ValueError(f"gated attention: {2 * self.cos.shape[1]} rotated dimensions do not fit a head of {spec.head_dim}")
        self.w_in = self.w_o = self.q_norm = self.k_norm = self.sink = self.mix = self.bias = self.o_bias = self.conv = self.q_mul = None

    @staticmethod
    def tensor_needs(spec: GatedAttentionSpec) -> List[TensorNeed]:
        H, G, dk, dv = spec.num_heads, spec.num_kv_heads, spec.head_dim, spec.value_dim
        out = [TensorNeed(spec.q_weight, (H * dk, spec.hidden)), TensorNeed(spec.o_weight, (spec.hidden, H * dv))]
        if spec.own_kv:
            out.append(TensorNeed(spec.k_weight, (G * dk, spec.hidden)))
            if not spec.keys_as_values:
                out.append(TensorNeed(spec.v_weight, (G * dv, spec.hidden)))
        for name, size in ((spec.q_bias, H * dk), (spec.k_bias if spec.own_kv else None, G * dk), (spec.v_bias if spec.own_kv else None, G * dv),
                           (spec.o_bias, spec.hidden)):
            if name:
                out.append(TensorNeed(name, (size,), "float32"))
        if spec.taps:
            for name, size in ((spec.q_conv, H * dk), (spec.k_conv, G * dk), (spec.v_conv, G * dv)):
                out.append(TensorNeed(name, (size, spec.taps), "float32"))
        if spec.gate_weight:
            out.append(TensorNeed(spec.gate_weight, (H if spec.gate_per_head else H * dv, spec.hidden)))
        wide = spec.norm_scope == "projection"
        for name, heads in ((spec.q_norm, H), (spec.k_norm, G)):
            if name:
                out.append(TensorNeed(name, (heads * dk if wide else dk,), "float32", init="around_one"))
        if spec.sink:
            out.append(TensorNeed(spec.sink, (H,), "float32"))
        if spec.value_mix_weight:  # read by "mix" layers; a "first" layer's file may carry one that nobody uses
            out.append(TensorNeed(spec.value_mix_weight, (), "float32"))
        return out + list(part_class("position", spec.position.kind).tensor_needs(spec.position))

    def subparts(self):
        return (self.position,)

    def cache_needs(self):
        s = self.spec
        if not s.own_kv:
            return ()
        kv = KVNeed(s.num_kv_heads, s.head_dim, s.window if s.cache_window is None else s.cache_window, value_dim=s.value_dim)
        if s.taps > 1:
            return (kv, StateNeed(CONV, (s.taps - 1, self._channels())))
        return (kv,)

    def _channels(self) -> int:
        s = self.spec
        return (s.num_heads + s.num_kv_heads) * s.head_dim + s.num_kv_heads * s.value_dim

    def kernel_notes(self):
        s, ops = self.spec, self.env.ops
        if self.env.dtype == torch.bfloat16 and hasattr(ops, "gated_attention_kernel"):
            kernel = ops.gated_attention_kernel(s.num_heads, s.num_kv_heads, s.head_dim, s.value_dim)
            if kernel != "tensor cores":
                return [f"gated attention with heads of {s.head_dim} / {s.value_dim} numbers: runs on {kernel}"]
        return []

    def load(self, tensors) -> None:
        s = self.spec
        rows = [tensors[s.q_weight]]
        if s.own_kv:
            rows += [tensors[s.k_weight]] + ([] if s.keys_as_values else [tensors[s.v_weight]])
        if s.gate_weight:
            rows.append(tensors[s.gate_weight])
        self.w_in = torch.cat(rows, dim=0).contiguous()  # one product for everything that reads the mixer's input
        self.w_o = tensors[s.o_weight]
        self.q_norm = tensors[s.q_norm] if s.q_norm else None
        self.k_norm = tensors[s.k_norm] if s.k_norm else None
        self.sink = tensors[s.sink] if s.sink else None
        if s.sink_score is not None:
            self.sink = torch.full((s.num_heads,), float(s.sink_score), dtype=torch.float32, device=self.env.device)
        biases = [(s.q_bias, s.num_heads * s.head_dim)]
        if s.own_kv:
            biases.append((s.k_bias, s.num_kv_heads * s.head_dim))
            if s.v_bias:
                biases.append((s.v_bias, s.num_kv_heads * s.value_dim))
        if any(name for name, _ in biases):  # one vector over the columns [q | k] or [q | k | v], zeros where a projection has none
            self.bias = torch.cat([tensors[name] if name else torch.zeros(size, dtype=torch.float32, device=self.env.device)
                                   for name, size in biases]).contiguous()
        self.o_bias = tensors[s.o_bias].contiguous() if s.o_bias else None
        if s.taps:  # [taps, channels]: neighbouring channels read neighbouring words
            self.conv = torch.cat([tensors[s.q_conv], tensors[s.k_conv], tensors[s.v_conv]], dim=0).t().contiguous()
        if s.q_temperature is not None:
            self.q_mul = torch.from_numpy(query_temperatures(s.q_temperature)).to(self.env.device)
        self.mix = tensors[s.value_mix_weight].reshape(1) if s.value_mix == "mix" else None
        self.position.load(tensors)

    def forward(self, x, ctx, cache: LayerCache) -> Optional[torch.Tensor]:
        s, ops, n, dt = self.spec, self.env.ops, ctx.n_tokens, self.env.dtype
        if isinstance(x, NormalizedRows):
            x = x.dense(ctx)
        H, G, dk, dv = s.num_heads, s.num_kv_heads, s.head_dim, s.value_dim
        if cache.k is None or (not s.own_kv and cache.writes):
            raise RuntimeError("gated attention: this layer has no keys and values of its own, and its run names no cache to read")
        if n <= 64:
            parts = ops.gemm_partials(x[:n], self.w_in, ctx.ws, "gated_attention.in_parts")
        else:
            parts = ctx.ws.get("gated_attention.in_parts", (1, n, self.w_in.shape[0]), torch.float32)
            ops.gemm(x[:n], self.w_in, parts[0])
        role, v_first = 0, None
        if s.value_mix is not None:
            shared = ctx.shared
            if s.value_mix == "first":
                role = 1
                v_first = shared[V_FIRST] = ctx.ws.get(V_FIRST, (n, G * dv), torch.float32)
            else:
                role, v_first = 2, shared.get(V_FIRST)
                if v_first is None or v_first.shape[1] != G * dv:
                    raise RuntimeError("gated attention: a layer mixes values in, but no earlier layer of the step left values of its shape")
        q = ctx.ws.get("gated_attention.q", (n, H * dk), dt)
        writes = cache.writes and cache.k is not None and s.own_kv
        wide = {"norm_wide": True} if s.norm_scope == "projection" else {}
        if self.row_form:
            wide.update(bias=self.bias, neighbours=s.rot_pairs == "neighbours", conv=self.conv, conv_state=cache.states[CONV] if s.taps > 1 else None,
                        q_mul=self.q_mul)
        elif self.bias is not None or s.unit_rms or s.rot_pairs != "half" or s.keys_as_values:
            wide = {"bias": self.bias, "unit_rms": s.unit_rms, "neighbours": s.rot_pairs == "neighbours", "keys_as_values": s.keys_as_values}
        ops.qkv_prep(parts, H, G if s.own_kv else 0, dk, dv, self.q_norm, self.k_norm, s.eps, self.cos, self.sin, ctx, ctx.block_tables[cache.group], q,
                     cache.k if writes else None, cache.v if writes else None, role, self.mix, v_first, **wide)
        att = ctx.ws.get("gated_attention.out", (n, H * dv), dt)
        g_off = H * dk + (G * dk + (0 if s.keys_as_values else G * dv) if s.own_kv else 0)
        ops.gated_attention(q, cache.k, cache.v, ctx, ctx.block_tables[cache.group], att, H, G, dk, dv, s.scale, s.window, s.chunk,
                            self.sink, parts if s.gate_weight else None, g_off, **({"gate_per_head": True} if s.gate_per_head else {}))
        if self.o_bias is None:
            return add_into_stream_or_partials(ops, att, self.w_o, ctx, False, "gated_attention.delta")
        keep, ctx.residual = ctx.residual, None  # the sums are wanted here: the bias goes with them
        delta = add_into_stream_or_partials(ops, att, self.w_o, ctx, False, "gated_attention.delta")
        ctx.residual = keep
        if ctx.takes_delta_bias:
            ctx.delta_bias = self.o_bias  # the block adds it with the sums
        else:
            ops.stream_add(delta if delta.dim() == 2 else delta[0], None, n_rows=n, bias=self.o_bias)
        return delta


register_part("mixer", "gated_attention", GatedAttention)
