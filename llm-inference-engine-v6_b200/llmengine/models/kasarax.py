"""The Kasarax decoder ("architecture": "Kasarax") as a description in parts.

Tensors: `embed` [vocab, width] (also the output head), `final.norm`; per layer i `l<i>.norm1`; an attention mixer's
`l<i>.mix.{q, q.b, k, k.b, v, v.b, g, o, o.b}`; a parallel mixer's `l<i>.mix.left.{q, k, v, q.conv, k.conv, v.conv, q.norm, k.norm, sink,
o, out}` beside `l<i>.mix.right.{q, k, v, g, norm, o, out}`; a dense feed-forward's `l<i>.mlp.{gate, up, down}` or a routed one's
`l<i>.mlp.{router, e<k>.up, e<k>.down}`.

A layer is a parallel block with ONE norm (weight 1 + w): h += mixer(norm1(h)) + ff(norm1(h)). The parallel mixer is a pair: attention
behind short convolutions beside linear attention with a fixed decay a head, the mean of the two results after a norm each. Logits are
the embedding table's, times a constant that the final norm carries.
"""
from __future__ import annotations

from ..config.kasarax import DenseFF, KasaraxConfig, MoEFF, sizes_from_tensors
from ..config.registry import Architecture, register_architecture
from ..parts.spec import (BlockSpec, EmbeddingSpec, GatedAttentionSpec, GatedMLPSpec, GroupRoutedMLPSpec, HeadSpec, LayerRun,
                          LightningAttentionSpec, MixerPairSpec, ModelSpec, NormSpec, QueryTemperatureSpec, ScaledRotarySpec)


def describe_kasarax(cfg: KasaraxConfig) -> ModelSpec:
    layers = []

    def norm(name, gain=1.0):
        return NormSpec("rmsnorm_unit_offset", cfg.width, cfg.eps, name, gain)

    def rotation(dims, base):
        return ScaledRotarySpec(kind="rope_ramp", dims=dims, base=base, max_positions=cfg.max_positions)

    for i, l in enumerate(cfg.layers):
        p, m = f"l{i}.", l.mixer
        q = p + "mix."
        if l.type == "attention":
            temp = None if m.q_temp is None else QueryTemperatureSpec(m.q_temp.coef, m.q_temp.every, cfg.max_positions)
            mixer = GatedAttentionSpec(kind="gated_attention", hidden=cfg.width, num_heads=m.heads, num_kv_heads=m.kv_heads, head_dim=m.dim,
                                       value_dim=m.vdim, scale=m.scale, eps=cfg.eps, position=rotation(0, 10000.0), q_weight=q + "q",
                                       k_weight=q + "k", v_weight=q + "v", o_weight=q + "o", q_bias=q + "q.b", k_bias=q + "k.b",
                                       v_bias=q + "v.b", o_bias=q + "o.b", gate_weight=q + "g", gate_per_head=True, sink_score=0.0,
                                       q_temperature=temp)
        else:
            a, r, lp, rp = m.left, m.right, q + "left.", q + "right."
            left = GatedAttentionSpec(kind="gated_attention", hidden=cfg.width, num_heads=a.heads, num_kv_heads=a.kv_heads, head_dim=a.dim,
                                      value_dim=a.vdim, scale=a.scale, eps=cfg.eps, position=rotation(a.rot_dims, a.rot_base),
                                      q_weight=lp + "q", k_weight=lp + "k", v_weight=lp + "v", o_weight=lp + "o", q_norm=lp + "q.norm",
                                      k_norm=lp + "k.norm", norm_scope="projection", rot_pairs="neighbours", sink=lp + "sink",
                                      taps=a.taps, q_conv=lp + "q.conv", k_conv=lp + "k.conv", v_conv=lp + "v.conv")
            right = LightningAttentionSpec(kind="lightning_attention", hidden=cfg.width, heads=r.heads, dim=r.dim, vdim=r.vdim, decay=r.decay,
                                           eps=cfg.eps, q_weight=rp + "q", k_weight=rp + "k", v_weight=rp + "v", g_weight=rp + "g",
                                           norm_weight=rp + "norm", o_weight=rp + "o")
            mixer = MixerPairSpec(kind="mixer_pair", hidden=cfg.width, left=left, right=right, combine="normed_mean", left_norm=lp + "out",
                                  right_norm=rp + "out", eps=cfg.eps)
        f, ff = l.mlp, None
        if isinstance(f, DenseFF):
            ff = GatedMLPSpec(kind="gated_mlp", hidden=cfg.width, intermediate=f.ff, gate_weight=p + "mlp.gate", up_weight=p + "mlp.up",
                              down_weight=p + "mlp.down", activation="silu")
        elif isinstance(f, MoEFF):
            ff = GroupRoutedMLPSpec(kind="group_routed_mlp", hidden=cfg.width, intermediate=f.ff, experts=f.experts, top=f.top,
                                    router_weight=p + "mlp.router", correction=None, gate_weights=(),
                                    up_weights=tuple(f"{p}mlp.e{k}.up" for k in range(f.experts)),
                                    down_weights=tuple(f"{p}mlp.e{k}.down" for k in range(f.experts)),
                                    activation="relu_squared", score="sigmoid", normalize=False, weigh="input")
        layers.append(BlockSpec(kind="parallel", norm1=norm(p + "norm1"), mixer=mixer, norm2=None, feed_forward=ff))
    return ModelSpec(
        architecture=cfg.architecture,
        embedding=EmbeddingSpec("embed", cfg.vocab, cfg.width),
        layers=tuple(layers),
        order=tuple(LayerRun(i) for i in range(len(layers))),
        final_norm=norm("final.norm", cfg.logit_scale),
        head=HeadSpec("embed", cfg.vocab, cfg.width),
        max_positions=cfg.max_positions,
        eos_token_ids=cfg.eos_token_ids,
    )


KASARAX = Architecture(name="Kasarax", parse_config=KasaraxConfig.from_dict, describe=describe_kasarax,
                       config_to_json=lambda cfg: cfg.to_dict(), sizes_from_tensors=sizes_from_tensors)
register_architecture(KASARAX, replace=True)
