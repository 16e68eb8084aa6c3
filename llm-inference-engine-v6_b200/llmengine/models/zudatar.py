"""The Zudatar decoder ("architecture": "Zudatar") as a description in parts.

Tensors: `embed` [vocab, width] (also the output head), `bigram` [buckets + 1, width], `final.norm`; per layer i `l<i>.norm1`,
`l<i>.norm1b` and, with a feed-forward, `l<i>.norm2`, `l<i>.norm2b` and `l<i>.mlp.{gate, up, down}`; a delta mixer's
`l<i>.mix.{q, k, v, q.conv, k.conv, v.conv, b, A_log, norm, a1, a2, dt_bias, g1, g2, o}`; an attention mixer's
`l<i>.mix.{q, q.b, k, k.b, g, o}`; a latent-attention mixer's `l<i>.mix.{dq, dq.norm, uq, dkv, dkv.norm, uk, uv, sink, g, o}` (a
layer that reads another layer's latents has no `dkv` and `dkv.norm`).

The stream starts as embed[token] * scale plus a row of the pair table chosen by the previous token and this one. A layer is a
sandwich block: h += norm1b(mixer(norm1(h))); h += norm2b(ff(norm2(h))). Logits are the embedding table's, times a constant that
the final norm carries.
"""
from __future__ import annotations

from ..config.registry import Architecture, register_architecture
from ..config.zudatar import ZudatarConfig, sizes_from_tensors
from ..parts.spec import (BlockSpec, ChannelDeltaSpec, EmbeddingSpec, GatedAttentionSpec, GatedMLPSpec, HeadSpec, LatentAttentionSpec,
                          LayerRun, ModelSpec, NormSpec, ScaledRotarySpec)

UNIT_EPS = 1e-6  # under the root when the delta rule's queries and keys are made unit vectors


def kept_window(cfg: ZudatarConfig, owner: int) -> int:
    """How many of the last latents layer `owner`'s cache must keep: the widest window among the layer itself and the layers that
    read its latents (0, everything, as soon as one of them has no window)."""
    windows = [cfg.layers[owner].mixer.window] + [l.mixer.window for l in cfg.layers if l.type == "latent_attention" and l.mixer.kv_from == owner]
    return 0 if 0 in windows else max(windows)


def describe_zudatar(cfg: ZudatarConfig) -> ModelSpec:
    layers, order, ignore = [], [], []

    def norm(name, gain=1.0):
        return NormSpec("rmsnorm", cfg.width, cfg.eps, name, gain)

    def rotation(dims, base):
        return ScaledRotarySpec(kind="rope_ramp", dims=dims, base=base, max_positions=cfg.max_positions)

    for i, l in enumerate(cfg.layers):
        p, m = f"l{i}.", l.mixer
        q = p + "mix."
        source = None
        if l.type == "channel_delta":
            mixer = ChannelDeltaSpec(kind="channel_delta", hidden=cfg.width, heads=m.heads, kv_heads=m.kv_heads, dim=m.dim, vdim=m.vdim,
                                     taps=m.taps, decay_rank=m.decay_rank, gate_rank=m.gate_rank, eps=cfg.eps, q_weight=q + "q",
                                     k_weight=q + "k", v_weight=q + "v", q_conv=q + "q.conv", k_conv=q + "k.conv", v_conv=q + "v.conv",
                                     b_weight=q + "b", a1_weight=q + "a1", a2_weight=q + "a2", a_log=q + "A_log", dt_bias=q + "dt_bias",
                                     g1_weight=q + "g1", g2_weight=q + "g2", norm_weight=q + "norm", o_weight=q + "o", unit_eps=UNIT_EPS)
        elif l.type == "attention":
            mixer = GatedAttentionSpec(kind="gated_attention", hidden=cfg.width, num_heads=m.heads, num_kv_heads=m.kv_heads, head_dim=m.dim,
                                       value_dim=m.vdim, scale=m.scale, eps=cfg.eps, position=rotation(m.rot_dims, m.rot_base),
                                       q_weight=q + "q", k_weight=q + "k", v_weight=None, o_weight=q + "o", q_bias=q + "q.b", k_bias=q + "k.b",
                                       gate_weight=q + "g", gate_per_head=True, window=m.window, rot_pairs="neighbours", unit_rms=True,
                                       keys_as_values=True)
        else:
            source, own = m.kv_from, m.kv_from is None
            mixer = LatentAttentionSpec(kind="latent_attention", hidden=cfg.width, heads=m.heads, dim=m.dim, rot_dim=0, vdim=m.vdim,
                                        kv_rank=m.kv_rank, q_rank=m.q_rank, scale=m.scale, eps=cfg.eps, position=rotation(0, 10000.0),
                                        dq_weight=q + "dq", dq_norm=q + "dq.norm", uq_weight=q + "uq", dkv_weight=q + "dkv" if own else None,
                                        dkv_norm=q + "dkv.norm" if own else None, uk_weight=q + "uk", uv_weight=q + "uv", gate_weight=q + "g",
                                        o_weight=q + "o", window=m.window, sink=q + "sink", gate_per_head=True, own_kv=own,
                                        cache_window=kept_window(cfg, i) if own else None)
        order.append(LayerRun(i, cache_from=source))  # every layer runs once, so a layer's index is its run's
        ff = norm2 = norm2_out = None
        if l.mlp is None:
            ignore += [p + "norm2", p + "norm2b"]  # a layer without a feed-forward has no use for them
        else:
            norm2, norm2_out = norm(p + "norm2"), norm(p + "norm2b")
            ff = GatedMLPSpec(kind="gated_mlp", hidden=cfg.width, intermediate=l.mlp.ff, gate_weight=p + "mlp.gate", up_weight=p + "mlp.up",
                              down_weight=p + "mlp.down", activation="silu")
        layers.append(BlockSpec(kind="sandwich", norm1=norm(p + "norm1"), mixer=mixer, norm2=norm2, feed_forward=ff,
                                norm1_out=norm(p + "norm1b"), norm2_out=norm2_out))
    b = cfg.pairs
    pair = {} if b is None else {"kind": "lookup_pairs", "pair_weight": "bigram", "pair_buckets": b.buckets, "pair_mul_prev": b.mul_prev,
                                 "pair_mul_cur": b.mul_cur}
    return ModelSpec(
        architecture=cfg.architecture,
        embedding=EmbeddingSpec("embed", cfg.vocab, cfg.width, scale=cfg.embed_scale, **pair),
        layers=tuple(layers),
        order=tuple(order),
        final_norm=norm("final.norm", cfg.logit_scale),
        head=HeadSpec("embed", cfg.vocab, cfg.width),
        max_positions=cfg.max_positions,
        eos_token_ids=cfg.eos_token_ids,
        ignore=tuple(ignore),
    )


ZUDATAR = Architecture(name="Zudatar", parse_config=ZudatarConfig.from_dict, describe=describe_zudatar,
                       config_to_json=lambda cfg: cfg.to_dict(), sizes_from_tensors=sizes_from_tensors)
register_architecture(ZUDATAR, replace=True)
