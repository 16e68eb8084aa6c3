"""Tiny Zudatar configurations and their weights for the tests. The configurations differ from one another in every size and
option, and no two sizes that could be mixed up are equal within one of them (query heads != key/value heads, key size != value
size where the design leaves both free, rotated part != head, window != page, taps != rank, the two low-rank maps' ranks apart).

The weights are made here by rules of the test's own (not the package's random-weights mode), so that every tensor matters: norm
weights around one, biases, sinks and pair rows large enough to show, decays from fast to very slow (a state that is lost or reset
shows hundreds of tokens later). `sharp=True` scales the queries so that the softmax of most heads rests on one or two keys,
wherever they are: a key that is lost, shifted, read from a wrong page or let through a window's edge moves the logits."""
from __future__ import annotations

import json
import math
import os

import torch


def delta(heads, kv_heads, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def att(heads, kv_heads, dim, scale, window, rot=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale, "mask": {"size": window}}
    if rot:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
    return m


def lat(heads, dim, vdim, kv_rank, q_rank, scale, window, kv_from=None):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": scale, "mask": {"size": window}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def layer(kind, mixer, ff=None):
    return {"type": kind, "mixer": mixer, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(vocab, width, eps, scale, pairs, logit_scale, layers, max_positions=512):
    return {"architecture": "Zudatar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": logit_scale, "max_positions": max_positions,
            "embedding": {"scale": scale, "bigram": {"buckets": pairs[0], "mul_prev": pairs[1], "mul_cur": pairs[2]}}, "layers": layers}


# ranks of the low-rank maps (decay, gate): no keys of config.json; make_tensors draws the maps with these first dimensions
RANKS = {"za": {1: (5, 7), 4: (3, 2)}, "zb": {0: (32, 40), 3: (8, 16)}, "zc": {2: (1, 9)}}

# A: nothing a multiple of 8; latent attention first and last, the last one on the first one's latents through a WIDER window; shared
#    query/key heads in one delta layer, a single tap in the other; pages of 4
ZUDATAR_A = config(301, 72, 1e-5, 3.7, (53, 17, 5), 1.9, [
    layer("latent_attention", lat(3, 10, 14, 18, 22, 0.4, 7), 44),
    layer("channel_delta", delta(4, 2, 12, 10, 3), 20),
    layer("attention", att(6, 2, 18, 0.21, 13, (8, 777.0))),
    layer("latent_attention", lat(2, 12, 6, 18, 9, 0.35, 21, kv_from=0), 28),
    layer("channel_delta", delta(3, 3, 18, 6, 1))])
# B: sizes the tensor-core products and attention take (latents of 64 and 128, heads of 32 / 64 / 128); a borrower with a NARROWER
#    window; a value size of its own; pages of 16
ZUDATAR_B = config(512, 128, 1e-6, 8.0, (769, 31, 113), 0.6, [
    layer("channel_delta", delta(4, 2, 32, 64, 4), 256),
    layer("attention", att(4, 2, 64, 0.15, 48, (24, 20000.0)), 384),
    layer("latent_attention", lat(6, 32, 48, 64, 40, 0.2, 40), 128),
    layer("channel_delta", delta(2, 2, 64, 32, 2)),
    layer("latent_attention", lat(4, 64, 32, 64, 72, 0.15, 17, kv_from=2), 256),
    layer("attention", att(5, 1, 32, 0.18, 24))])
# C: one key/value head for five query heads, a window of one page, a window of a single key, two borrowers of one owner, a rank of
#    one, one bucket, no rotation in one layer and a whole head's in another; pages of 8
ZUDATAR_C = config(97, 48, 1e-5, 1.0, (1, 3, 2), 1.0, [
    layer("attention", att(5, 1, 16, 0.4, 8, (16, 300.0)), 40),
    layer("latent_attention", lat(1, 8, 20, 12, 6, 0.5, 1), 24),
    layer("channel_delta", delta(2, 1, 20, 12, 2), 16),
    layer("latent_attention", lat(4, 16, 4, 12, 14, 0.3, 30, kv_from=1)),
    layer("attention", att(3, 3, 10, 0.35, 5), 32),
    layer("latent_attention", lat(2, 6, 10, 12, 10, 0.45, 12, kv_from=1), 24)], 400)

ZUDATAR = {"za": (ZUDATAR_A, 4), "zb": (ZUDATAR_B, 16), "zc": (ZUDATAR_C, 8)}  # name -> (config.json, page size)


def ranks_of(cfg):
    for name, (c, _) in ZUDATAR.items():
        if c is cfg:
            return RANKS[name]
    return {}


def make_tensors(cfg, seed, dtype, sharp=False, ranks=None):
    """name -> tensor, as a checkpoint stores them (everything in `dtype`: the reader widens what it wants wider)."""
    g = torch.Generator().manual_seed(seed)
    D, V = cfg["width"], cfg["vocab"]
    ranks = ranks_of(cfg) if ranks is None else ranks
    e = cfg["embedding"]
    t = {}

    def lin(name, out, inp, gain=1.0):
        t[name] = torch.randn(out, inp, generator=g) * (gain / math.sqrt(inp))

    def near_one(name, n, spread=0.2):
        t[name] = 1.0 + spread * torch.randn(n, generator=g)

    t["embed"] = torch.randn(V, D, generator=g) * 0.5
    t["bigram"] = torch.randn(e["bigram"]["buckets"] + 1, D, generator=g) * (0.4 * e["scale"])  # as large as the tokens' own rows
    near_one("final.norm", D)
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        q = p + "mix."
        near_one(p + "norm1", D)
        near_one(p + "norm1b", D)
        if l["type"] == "channel_delta":
            H, G, dk, dv, K = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
            ra, rg = ranks.get(i, (16, 16))
            lin(q + "q", G * dk, D); lin(q + "k", G * dk, D); lin(q + "v", H * dv, D); lin(q + "o", D, H * dv)
            for s, c in (("q", G * dk), ("k", G * dk), ("v", H * dv)):
                t[q + s + ".conv"] = torch.randn(c, K, generator=g) * (0.8 / math.sqrt(K))
            lin(q + "b", H, D, gain=1.5)
            lin(q + "a1", ra, D); lin(q + "a2", H * dk, ra, gain=0.7)
            lin(q + "g1", rg, D); lin(q + "g2", H * dv, rg, gain=2.0)
            t[q + "A_log"] = torch.rand(H, generator=g) * math.log(200.0) + math.log(0.01)          # exp(A_log): 0.01 .. 2
            step = torch.exp(torch.rand(H * dk, generator=g) * math.log(50.0) + math.log(0.02))      # softplus(dt_bias): 0.02 .. 1
            t[q + "dt_bias"] = torch.log(torch.expm1(step))
            near_one(q + "norm", dv)
        elif l["type"] == "attention":
            H, G, dk = m["heads"], m["kv_heads"], m["dim"]
            lin(q + "q", H * dk, D); lin(q + "k", G * dk, D); lin(q + "o", D, H * dk); lin(q + "g", H, D, gain=2.0)
            t[q + "q.b"] = 0.5 * torch.randn(H * dk, generator=g)
            t[q + "k.b"] = 0.5 * torch.randn(G * dk, generator=g)
            # (queries and keys have unit root mean squares, so their scores' spread is scale * sqrt(dk) whatever the weights; the
            # configurations' scales set it, and sharp tests raise them)
        else:
            H, dk, dv, R, Rq = m["heads"], m["dim"], m["vdim"], m["kv_rank"], m["q_rank"]
            lin(q + "dq", Rq, D); near_one(q + "dq.norm", Rq, 0.3)
            lin(q + "uq", H * dk, Rq, gain=(6.0 if sharp else 1.0) / (m["scale"] * math.sqrt(dk)))
            if m.get("kv_from") is None:
                lin(q + "dkv", R, D); near_one(q + "dkv.norm", R, 0.3)
            lin(q + "uk", H * dk, R); lin(q + "uv", H * dv, R); lin(q + "o", D, H * dv); lin(q + "g", H, D, gain=2.0)
            t[q + "sink"] = 1.0 + 1.5 * torch.randn(H, generator=g)
        f = l.get("mlp")
        if f:
            near_one(p + "norm2", D)
            near_one(p + "norm2b", D)
            lin(p + "mlp.gate", f["ff"], D, gain=1.5); lin(p + "mlp.up", f["ff"], D, gain=1.5); lin(p + "mlp.down", D, f["ff"])
    return {k: v.to(dtype).contiguous() for k, v in t.items()}


def sharpened(cfg, spread=6.0):
    """The configuration with attention scales under which most heads rest on one or two keys."""
    import copy
    c = copy.deepcopy(cfg)
    for l in c["layers"]:
        if l["type"] == "attention":
            l["mixer"]["scale"] = spread / math.sqrt(l["mixer"]["dim"])
    return c


def write_model(path, cfg, dtype, seed=11, sharp=False, ranks=None):
    from llmengine.weights.safetensors_io import write_safetensors
    ranks = ranks_of(cfg) if ranks is None else ranks
    if sharp:
        cfg = sharpened(cfg)
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(path, "model.safetensors"), make_tensors(cfg, seed, dtype, sharp, ranks))
    return path
