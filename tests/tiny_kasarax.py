"""Tiny Kasarax configurations and their weights for the tests. The configurations differ from one another in every size and
option, and no two sizes that could be mixed up are equal within one of them (query heads != key/value heads, key size != value
size, rotated part != head, attention heads != linear-attention heads, taps, experts, chosen experts, inner sizes).

The weights are made here by rules of the test's own (not the package's random-weights mode), so that every tensor matters: biases
and sinks large enough to show, norm weights spread, convolutions whose every tap counts, decays from fast to very slow (a state that
is lost or reset shows hundreds of tokens later), router logits far apart. `sharp=True` scales queries so that the softmax of most
heads rests on one or two keys, wherever they are: a key that is lost, shifted or read from a wrong page moves the logits."""
from __future__ import annotations

import json
import math
import os

import numpy as np
import torch


def att(heads, kv_heads, dim, vdim, scale, temp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if temp:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return m


def left(heads, kv_heads, dim, vdim, scale, conv, rot=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "conv": conv}
    if rot:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
    return m


def right(heads, dim, vdim, decay):
    return {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def layer(kind, mixer, mlp=None):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


def pair(a, b, mlp=None):
    return layer("parallel", {"left": a, "right": b}, mlp)


def config(vocab, width, eps, logit_scale, layers, max_positions=512):
    return {"architecture": "Kasarax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": logit_scale,
            "max_positions": max_positions, "layers": layers}


# A: nothing a multiple of 8; attention first and last; shared key/value heads on both kinds of attention; two of five experts; pages of 4
KASARAX_A = config(301, 70, 1e-5, 1.9, [
    layer("attention", att(6, 2, 18, 10, 0.25, (0.4, 7)), dense(44)),
    pair(left(4, 2, 12, 14, 0.3, 3, (8, 777.0)), right(3, 10, 6, (0.5, 0.97, 0.9995)), moe(22, 5, 2)),
    pair(left(3, 3, 10, 6, 0.35, 1), right(2, 7, 9, (1.0, 0.0))),
    layer("attention", att(5, 1, 14, 22, 0.2), moe(30, 3, 3))])
# B: sizes that the tensor-core products and attention take; heads of 32 / 64 / 128 in unequal pairs; four taps and two; one of six experts
KASARAX_B = config(512, 128, 1e-6, 0.6, [
    pair(left(4, 2, 64, 32, 0.15, 4, (24, 20000.0)), right(3, 32, 64, (0.9, 0.99, 0.999)), dense(256)),
    pair(left(6, 2, 32, 64, 0.2, 2, (32, 500.0)), right(2, 64, 48, (0.7, 0.995)), moe(96, 6, 1)),
    layer("attention", att(8, 2, 64, 128, 0.13, (0.3, 16)), moe(64, 4, 3)),
    layer("attention", att(4, 4, 32, 32, 0.2, (1.5, 100))),
    pair(left(5, 1, 128, 64, 0.1, 3, (2, 50.0)), right(1, 16, 32, (0.998,)), dense(384))])
# C: one key/value head for five query heads, five taps, a rotation over a whole head, as many experts as are chosen, steps of one
#    position in the query temperature, a layer without feed-forward; pages of 8
KASARAX_C = config(97, 48, 1e-4, 1.0, [
    pair(left(5, 1, 16, 8, 0.4, 5, (16, 300.0)), right(4, 6, 12, (0.3, 0.8, 0.99, 0.9999)), moe(20, 2, 2)),
    layer("attention", att(1, 1, 8, 20, 0.5, (0.7, 1)), moe(24, 7, 4)),
    pair(left(2, 2, 20, 12, 0.3, 2), right(1, 18, 5, (0.96,)), dense(40)),
    layer("attention", att(3, 3, 10, 6, 0.4, (2.0, 33)))], 400)

KASARAX = {"ka": (KASARAX_A, 4), "kb": (KASARAX_B, 16), "kc": (KASARAX_C, 8)}  # name -> (config.json, page size)


def make_tensors(cfg, seed, dtype, sharp=False):
    """name -> tensor, as a checkpoint stores them (everything in `dtype`: the reader widens what it wants wider)."""
    g = torch.Generator().manual_seed(seed)
    D, V = cfg["width"], cfg["vocab"]
    t = {}

    def lin(name, out, inp, gain=1.0):
        t[name] = torch.randn(out, inp, generator=g) * (gain / math.sqrt(inp))

    def vec(name, n, mean=0.0, spread=0.2):
        t[name] = mean + spread * torch.randn(n, generator=g)

    t["embed"] = torch.randn(V, D, generator=g)
    vec("final.norm", D)
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        q = p + "mix."
        vec(p + "norm1", D)
        if l["type"] == "attention":
            H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            lin(q + "q", H * dk, D, gain=(6.0 if sharp else 1.0) / (m["scale"] * math.sqrt(dk)))
            lin(q + "k", G * dk, D); lin(q + "v", G * dv, D); lin(q + "o", D, H * dv); lin(q + "g", H, D, gain=2.0)
            vec(q + "q.b", H * dk, spread=0.5); vec(q + "k.b", G * dk, spread=0.5); vec(q + "v.b", G * dv, spread=0.5); vec(q + "o.b", D, spread=0.5)
        else:
            a, r = m["left"], m["right"]
            H, G, dk, dv, K = a["heads"], a["kv_heads"], a["dim"], a["vdim"], a["conv"]
            for s, c in (("q", H * dk), ("k", G * dk), ("v", G * dv)):
                lin(f"{q}left.{s}", c, D)
                t[f"{q}left.{s}.conv"] = torch.randn(c, K, generator=g) * (1.0 / math.sqrt(K))
            # (queries and keys leave their norms with root mean squares of about one: the norm's weight sets the scores' spread)
            spread = (6.0 if sharp else 1.0) / (a["scale"] * math.sqrt(dk))
            t[q + "left.q.norm"] = spread * (1.0 + 0.3 * torch.randn(H * dk, generator=g))
            vec(q + "left.k.norm", G * dk, 1.0, 0.3)
            vec(q + "left.sink", H, 1.0, 1.5)
            lin(q + "left.o", D, H * dv)
            H, dk, dv = r["heads"], r["dim"], r["vdim"]
            lin(q + "right.q", H * dk, D, 1.5); lin(q + "right.k", H * dk, D, 1.5); lin(q + "right.v", H * dv, D, 1.5); lin(q + "right.g", H * dv, D, 2.0)
            vec(q + "right.norm", H * dv, 1.0, 0.3)
            lin(q + "right.o", D, H * dv)
            vec(q + "left.out", D, 1.0, 0.3); vec(q + "right.out", D, 1.0, 0.3)
        f = l.get("mlp")
        if f and f["kind"] == "dense":
            lin(p + "mlp.gate", f["ff"], D, gain=1.5); lin(p + "mlp.up", f["ff"], D, gain=1.5); lin(p + "mlp.down", D, f["ff"])
        elif f:
            lin(p + "mlp.router", f["router"]["experts"], D, gain=2.0)
            for e in range(f["router"]["experts"]):
                lin(f"{p}mlp.e{e}.up", f["expert"]["ff"], D, gain=1.5); lin(f"{p}mlp.e{e}.down", D, f["expert"]["ff"])
    return {k: v.to(dtype).contiguous() for k, v in t.items()}


def decided_ids(cfg, w, n, seed, gap=0.1):
    """n random token ids on which no router of the plain model has a close call: at every position tokens are drawn until each routed
    layer's last chosen and first unchosen logits lie `gap` apart (rounding in 16 bits moves them by a tenth of that). w: float64."""
    import plain_kasarax as P
    rng = np.random.default_rng(seed)
    m, ids = P.Plain(cfg, w), []

    def saved(st):
        return {k: saved(v) if isinstance(v, dict) else len(v) if isinstance(v, list) else v for k, v in st.items()}

    def put_back(st, old):
        for k in list(st):
            if k not in old:
                del st[k]
            elif isinstance(st[k], dict):
                put_back(st[k], old[k])
            elif isinstance(st[k], list):
                del st[k][old[k]:]
            else:
                st[k] = old[k]

    try:
        while len(ids) < n:
            old = [saved(st) for st in m.st]
            ids.append(int(rng.integers(0, cfg["vocab"])))
            P.GAPS = []
            m.run(ids[-1:])
            if any(float(g.min()) < gap for g in P.GAPS):
                ids.pop()
                for st, o in zip(m.st, old):
                    put_back(st, o)
    finally:
        P.GAPS = None
    return ids


def write_model(path, cfg, dtype, seed=11, sharp=False):
    from llmengine.weights.safetensors_io import write_safetensors
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(path, "model.safetensors"), make_tensors(cfg, seed, dtype, sharp))
    return path
