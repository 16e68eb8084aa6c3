"""A plain, slow implementation of the Zudatar decoder, one function per mechanism, in float64 (or any torch dtype) on the CPU.
It shares no code with the package: it takes config.json as a dict and the tensors by name and loops over tokens and heads.
The engine's tests compare against it.

Notation: T tokens, D width, H heads, G key/value heads, dk query/key size of a head, dv value size of a head. A layer is
    x += rms(mixer(rms(x) * n1)) * n1b;   x += rms(ff(rms(x) * n2)) * n2b     (the second line only with a feed-forward)
Every function that keeps something between calls takes a dict `st` and leaves what the next call needs there, so whole prompts,
portions and single tokens all go through the same code."""
from __future__ import annotations

import json
import math
import os
import struct

import numpy as np
import torch


# ---------------------------------------------------------------------------- files
def read_safetensors(path):
    with open(path, "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        head = json.loads(f.read(n))
        base = 8 + n
        out = {}
        for name, info in head.items():
            if name == "__metadata__":
                continue
            lo, hi = info["data_offsets"]
            f.seek(base + lo)
            raw = f.read(hi - lo)
            dt = info["dtype"]
            if dt == "BF16":
                a = np.frombuffer(raw, dtype="<u2").astype(np.uint32) << 16
                t = torch.from_numpy(a.view(np.float32).copy())
            elif dt == "F32":
                t = torch.from_numpy(np.frombuffer(raw, dtype="<f4").copy())
            else:
                raise ValueError(f"{name}: dtype {dt}")
            out[name] = t.reshape(info["shape"])
    return out


def read_model(model_dir, dtype=torch.float64):
    with open(os.path.join(model_dir, "config.json")) as f:
        cfg = json.load(f)
    w = read_safetensors(os.path.join(model_dir, "model.safetensors"))
    return cfg, {k: v.to(dtype) for k, v in w.items()}


# ---------------------------------------------------------------------------- small pieces
ROUNDING = None  # a function, or None. A 16-bit engine rounds the operands of its matrix products (a sublayer's input, queries, keys,
# values and latents, what enters an output projection); with ROUNDING set, the same happens here, everything else staying in the
# precision of the weights: the difference to a run without it is the error that rounding alone causes.


def _r(x):
    return x if ROUNDING is None else ROUNDING(x)


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.where(z > 30, z, torch.log1p(torch.exp(torch.clamp(z, max=30))))


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def first_visible(pos, window):
    """The oldest position that a token at `pos` sees through a window of `window` tokens that counts the token itself."""
    return max(0, pos - window + 1)


# ---------------------------------------------------------------------------- embedding
def embedding(tokens, w, e, st):
    """scale * row of the token, plus a row of the pair table: (previous * mul_prev + token * mul_cur) mod buckets, or for a sequence's
    first token the row behind the buckets. st keeps the previous token."""
    b = e["bigram"]
    rows = []
    for t in tokens:
        t = int(t)
        prev = st.get("previous")
        row = b["buckets"] if prev is None else (prev * b["mul_prev"] + t * b["mul_cur"]) % b["buckets"]
        rows.append(w["embed"][t] * e["scale"] + w["bigram"][row])
        st["previous"] = t
    return torch.stack(rows)


# ---------------------------------------------------------------------------- delta rule with a decay per key channel
def short_conv_silu(x, weight, st, key):
    """x [T, C], weight [C, taps]: silu(sum_j weight[:, j] * x[t - (taps - 1) + j]); inputs before the sequence's first are zero; st
    keeps the last taps - 1 inputs."""
    taps = weight.shape[1]
    tail = st.get(key)
    if tail is None:
        tail = torch.zeros(taps - 1, x.shape[1], dtype=x.dtype)
    padded = torch.cat([tail, x], dim=0)
    out = torch.stack([(padded[t:t + taps] * weight.t()).sum(0) for t in range(x.shape[0])])
    st[key] = padded[padded.shape[0] - (taps - 1):] if taps > 1 else tail
    return silu(out)


def channel_decay(h, w, p, H, dk):
    """[T, H, dk]: exp(-exp(A_log of the head) * softplus(W_a2 W_a1 h + dt_bias)), a number per head and key channel."""
    z = (h @ w[p + "a1"].t()) @ w[p + "a2"].t() + w[p + "dt_bias"]
    return torch.exp(-torch.exp(w[p + "A_log"])[None, :, None] * softplus(z).view(-1, H, dk))


def delta_step(S, q, k, v, g, beta):
    """One token through the state of all heads. S [H, dk, dv]; q, k, g [H, dk]; v [H, dv]; beta [H] -> (S, o [H, dv])."""
    S = S * g[:, :, None]
    u = beta[:, None] * (v - torch.einsum("hkv,hk->hv", S, k))
    S = S + k[:, :, None] * u[:, None, :]
    return S, torch.einsum("hkv,hk->hv", S, q)


def channel_delta(h, w, p, m, eps, st):
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = short_conv_silu(h @ w[p + "q"].t(), w[p + "q.conv"], st, "cq").view(T, G, dk)
    k = short_conv_silu(h @ w[p + "k"].t(), w[p + "k.conv"], st, "ck").view(T, G, dk)
    v = short_conv_silu(h @ w[p + "v"].t(), w[p + "v.conv"], st, "cv").view(T, H, dv)
    shared = [a // (H // G) for a in range(H)]   # which query/key head a head uses
    q, k = unit(q)[:, shared] * dk ** -0.5, unit(k)[:, shared]
    beta = sigmoid(h @ w[p + "b"].t())
    g = channel_decay(h, w, p, H, dk)
    gate = sigmoid((h @ w[p + "g1"].t()) @ w[p + "g2"].t()).view(T, H, dv)
    S = st.get("S")
    if S is None:
        S = torch.zeros(H, dk, dv, dtype=h.dtype)
    out = []
    for t in range(T):
        S, o = delta_step(S, q[t], k[t], v[t], g[t], beta[t])
        out.append((rms(o, eps) * w[p + "norm"] * gate[t]).reshape(-1))
    st["S"] = S
    return _r(torch.stack(out)) @ w[p + "o"].t()


# ---------------------------------------------------------------------------- attention whose values are its keys
def rotate_neighbours(x, pos, rot):
    """x [heads, dk]: numbers 2i and 2i + 1 of the first rot.dims of a head turn together by pos * base^(-2i/dims)."""
    if not rot or not rot["dims"]:
        return x
    d = rot["dims"]
    out = x.clone()
    for i in range(d // 2):
        a = pos * float(rot["base"]) ** (-2.0 * i / d)
        c, s = math.cos(a), math.sin(a)
        u, v = x[:, 2 * i], x[:, 2 * i + 1]
        out[:, 2 * i] = u * c - v * s
        out[:, 2 * i + 1] = v * c + u * s
    return out


def attention(h, w, p, m, eps, st):
    """Keys and queries are rotated and then made of root mean square one; the values are the keys as they come from the projection."""
    H, G, dk = m["heads"], m["kv_heads"], m["dim"]
    T, pos0 = h.shape[0], st.get("n", 0)
    out = []
    for t in range(T):
        pos = pos0 + t
        q = (w[p + "q"] @ h[t] + w[p + "q.b"]).view(H, dk)
        k = (w[p + "k"] @ h[t] + w[p + "k.b"]).view(G, dk)
        st.setdefault("v", []).append(_r(k))
        q = _r(rms(rotate_neighbours(q, pos, m.get("rot")), eps))
        st.setdefault("k", []).append(_r(rms(rotate_neighbours(k, pos, m.get("rot")), eps)))
        lo = first_visible(pos, m["mask"]["size"])
        K, V = torch.stack(st["k"][lo:pos + 1]), torch.stack(st["v"][lo:pos + 1])
        gate = sigmoid(w[p + "g"] @ h[t])
        heads = []
        for a in range(H):
            b = a // (H // G)
            pr = torch.softmax((K[:, b] @ q[a]) * m["scale"], dim=0)
            heads.append(pr @ V[:, b] * gate[a])
        out.append(torch.cat(heads))
    st["n"] = pos0 + T
    return _r(torch.stack(out)) @ w[p + "o"].t()


# ---------------------------------------------------------------------------- latent attention with a sink
def softmax_with_sink(scores, sink):
    """exp(score) / (sum of exp(scores) + exp(sink)): the sink is one more term of the denominator and of nothing else."""
    top = torch.maximum(scores.max(), sink)
    e = torch.exp(scores - top)
    return e / (e.sum() + torch.exp(sink - top))


def latent_attention(h, w, p, m, eps, st, owner=None):
    """One latent a token for keys and values; owner: the st of the layer whose latents are read (None: the layer has its own)."""
    H, dk, dv = m["heads"], m["dim"], m["vdim"]
    T, pos0 = h.shape[0], st.get("n", 0)
    Wk, Wv = w[p + "uk"].view(H, dk, -1), w[p + "uv"].view(H, dv, -1)
    cs = st.setdefault("c", []) if owner is None else owner["c"]
    K, V = st.setdefault("K", []), st.setdefault("V", [])   # this layer's keys and values of every latent so far, [H, *] each
    out = []
    for t in range(T):
        pos = pos0 + t
        if owner is None:
            cs.append(_r(rms(w[p + "dkv"] @ h[t], eps) * w[p + "dkv.norm"]))
        q = _r(w[p + "uq"] @ _r(rms(w[p + "dq"] @ h[t], eps) * w[p + "dq.norm"])).view(H, dk)
        K.append(Wk @ cs[pos])
        V.append(Wv @ cs[pos])
        lo = first_visible(pos, m["mask"]["size"])
        k, v = torch.stack(K[lo:pos + 1]), torch.stack(V[lo:pos + 1])
        gate = sigmoid(w[p + "g"] @ h[t])
        heads = []
        for a in range(H):
            pr = softmax_with_sink(k[:, a] @ q[a] * m["scale"], w[p + "sink"][a])
            heads.append(pr @ v[:, a] * gate[a])
        out.append(torch.cat(heads))
    st["n"] = pos0 + T
    return _r(torch.stack(out)) @ w[p + "o"].t()


# ---------------------------------------------------------------------------- feed-forward and the model
def dense_ff(h, w, p):
    return _r(silu(h @ w[p + "gate"].t()) * (h @ w[p + "up"].t())) @ w[p + "down"].t()


class Plain:
    """One sequence: `run` takes its next tokens and returns their logits [T, vocab]."""

    def __init__(self, cfg, w):
        self.cfg, self.w = cfg, w
        self.st = [dict() for _ in cfg["layers"]]
        self.first = {}

    def run(self, tokens, after_layers=None):
        cfg, w, eps = self.cfg, self.w, self.cfg["norm"]["eps"]
        x = embedding(tokens, w, cfg["embedding"], self.first)
        for i, l in enumerate(cfg["layers"]):
            p, m, st = f"l{i}.", l["mixer"], self.st[i]
            h = _r(rms(x, eps) * w[p + "norm1"])
            if l["type"] == "channel_delta":
                y = channel_delta(h, w, p + "mix.", m, eps, st)
            elif l["type"] == "attention":
                y = attention(h, w, p + "mix.", m, eps, st)
            elif l["type"] == "latent_attention":
                src = m.get("kv_from")
                y = latent_attention(h, w, p + "mix.", m, eps, st, None if src is None else self.st[src])
            else:
                raise ValueError(l["type"])
            x = x + rms(y, eps) * w[p + "norm1b"]
            if l.get("mlp"):
                y = dense_ff(_r(rms(x, eps) * w[p + "norm2"]), w, p + "mlp.")
                x = x + rms(y, eps) * w[p + "norm2b"]
            if after_layers is not None:
                after_layers.append(x.clone())
        return _r(rms(x, eps) * w["final.norm"]) @ w["embed"].t() * cfg["logit_scale"]


def forward(cfg, w, tokens, after_layers=None):
    return Plain(cfg, w).run(tokens, after_layers)


def greedy(cfg, w, prompt, n_new):
    m = Plain(cfg, w)
    out = list(prompt)
    logits = m.run(prompt)
    for _ in range(n_new):
        out.append(int(torch.argmax(logits[-1])))
        logits = m.run(out[-1:])
    return out
