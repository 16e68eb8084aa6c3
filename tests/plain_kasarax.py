"""A plain, slow implementation of the Kasarax decoder, one function per mechanism, in float64 (or any torch dtype) on the CPU.
It shares no code with the package: it takes config.json as a dict and the tensors by name and loops over tokens and heads.
The engine's tests compare against it.

Notation: T tokens, D width, H heads, G key/value heads, dk query/key size of a head, dv value size of a head. A layer is
    h = rms(x) * (1 + n1);   x += mixer(h) + ff(h)          (the second term only with a feed-forward)
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
ROUNDING = None  # a function, or None. A 16-bit engine rounds the operands of its matrix products (a sublayer's input, queries, keys
# and values, what enters an output projection); with ROUNDING set, the same happens here, everything else staying in the precision
# of the weights: the difference to a run without it is the error that rounding alone causes.


GAPS = None  # a list, or None: every routed layer adds, a token, the distance between its last chosen and first unchosen router logit


def _r(x):
    return x if ROUNDING is None else ROUNDING(x)


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def square_of_relu(z):
    return torch.clamp(z, min=0) ** 2


# ---------------------------------------------------------------------------- attention: shared pieces
def softmax_with_term(scores, term):
    """exp(score) / (sum of exp(scores) + exp(term)): the term enlarges the denominator and has no value."""
    top = torch.maximum(scores.max(), term)
    e = torch.exp(scores - top)
    return e / (e.sum() + torch.exp(term - top))


def attend(q, K, V, scale, terms, H, G):
    """One token's query heads q [H, dk] over the keys K [S, G, dk] and values V [S, G, dv] -> [H, dv]; terms [H]."""
    out = []
    for a in range(H):
        b = a // (H // G)
        out.append(softmax_with_term((K[:, b] @ q[a]) * scale, terms[a]) @ V[:, b])
    return torch.stack(out)


# ---------------------------------------------------------------------------- attention without positions
def query_temperature(pos, t):
    """What the query at position pos is multiplied with: it grows by steps, a step every t["every"] positions."""
    if not t:
        return 1.0
    return 1.0 + t["coef"] * math.log(math.floor((pos + 1) / t["every"]) + 1.0)


def attention(h, w, p, m, eps, st):
    """Biases on all four projections, a query temperature, 1 + sum exp(score) below the line, one gate a head."""
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T, pos0 = h.shape[0], st.get("n", 0)
    zero = torch.zeros(H, dtype=h.dtype)   # a score of 0: exp(0) = 1
    K, V = st.setdefault("k", []), st.setdefault("v", [])
    out = []
    for t in range(T):
        pos = pos0 + t
        q = (w[p + "q"] @ h[t] + w[p + "q.b"]).view(H, dk) * query_temperature(pos, m.get("q_temp"))
        K.append(_r((w[p + "k"] @ h[t] + w[p + "k.b"]).view(G, dk)))
        V.append(_r((w[p + "v"] @ h[t] + w[p + "v.b"]).view(G, dv)))
        o = attend(_r(q), torch.stack(K), torch.stack(V), m["scale"], zero, H, G)
        out.append((o * sigmoid(w[p + "g"] @ h[t])[:, None]).reshape(-1))
    st["n"] = pos0 + T
    return _r(torch.stack(out)) @ w[p + "o"].t() + w[p + "o.b"]


# ---------------------------------------------------------------------------- attention behind short convolutions
def short_conv(x, weight, st, key):
    """x [T, C], weight [C, taps]: sum_j weight[:, j] * x[t - (taps - 1) + j]; inputs before the sequence's first are zero; st keeps
    the last taps - 1 inputs."""
    taps = weight.shape[1]
    tail = st.get(key)
    if tail is None:
        tail = torch.zeros(taps - 1, x.shape[1], dtype=x.dtype)
    padded = torch.cat([tail, x], dim=0)
    out = torch.stack([(padded[t:t + taps] * weight.t()).sum(0) for t in range(x.shape[0])])
    st[key] = padded[padded.shape[0] - (taps - 1):] if taps > 1 else tail
    return out


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


def conv_attention(h, w, p, m, eps, st):
    """q, k and v through a convolution each, one RMS norm over all of q and one over all of k, rotation, a learned sink a head."""
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T, pos0 = h.shape[0], st.get("n", 0)
    qc = short_conv(h @ w[p + "q"].t(), w[p + "q.conv"], st, "cq")
    kc = short_conv(h @ w[p + "k"].t(), w[p + "k.conv"], st, "ck")
    vc = short_conv(h @ w[p + "v"].t(), w[p + "v.conv"], st, "cv")
    K, V = st.setdefault("k", []), st.setdefault("v", [])
    out = []
    for t in range(T):
        pos = pos0 + t
        q = rotate_neighbours((rms(qc[t], eps) * w[p + "q.norm"]).view(H, dk), pos, m.get("rot"))
        K.append(_r(rotate_neighbours((rms(kc[t], eps) * w[p + "k.norm"]).view(G, dk), pos, m.get("rot"))))
        V.append(_r(vc[t].view(G, dv)))
        out.append(attend(_r(q), torch.stack(K), torch.stack(V), m["scale"], w[p + "sink"], H, G).reshape(-1))
    st["n"] = pos0 + T
    return _r(torch.stack(out)) @ w[p + "o"].t()


# ---------------------------------------------------------------------------- linear attention with fixed decays
def lightning_step(S, q, k, v, decay):
    """One token through the state of all heads. S [H, dk, dv]; q, k [H, dk]; v [H, dv]; decay [H] -> (S, o [H, dv])."""
    S = decay[:, None, None] * S + k[:, :, None] * v[:, None, :]
    return S, torch.einsum("hkv,hk->hv", S, q)


def lightning(h, w, p, m, eps, st):
    H, dk, dv = m["heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q, k = (silu(h @ w[p + s].t()).view(T, H, dk) for s in "qk")
    v = silu(h @ w[p + "v"].t()).view(T, H, dv)
    gate = sigmoid(h @ w[p + "g"].t())
    decay = torch.tensor(m["decay"], dtype=h.dtype)
    S = st.get("S")
    if S is None:
        S = torch.zeros(H, dk, dv, dtype=h.dtype)
    out = []
    for t in range(T):
        S, o = lightning_step(S, q[t], k[t], v[t], decay)
        out.append(rms(o.reshape(-1), eps) * w[p + "norm"] * gate[t])   # one norm over all heads together
    st["S"] = S
    return _r(torch.stack(out)) @ w[p + "o"].t()


def side_by_side(h, w, p, m, eps, st):
    """The two mixers' results, each over its root mean square and times its weight, and the mean of the two."""
    left = conv_attention(h, w, p + "left.", m["left"], eps, st.setdefault("left", {}))
    right = lightning(h, w, p + "right.", m["right"], eps, st.setdefault("right", {}))
    return 0.5 * (rms(left, eps) * w[p + "left.out"] + rms(right, eps) * w[p + "right.out"])


# ---------------------------------------------------------------------------- feed-forwards
def dense_ff(h, w, p):
    return _r(silu(h @ w[p + "gate"].t()) * (h @ w[p + "up"].t())) @ w[p + "down"].t()


def experts_ff(h, w, p, f):
    """Each token through the experts with the largest sigmoid scores; a score multiplies what its expert reads."""
    top = f["router"]["top"]
    scores = sigmoid(h @ w[p + "router"].t())
    if GAPS is not None and top < f["router"]["experts"]:
        z = torch.sort(h @ w[p + "router"].t(), dim=1, descending=True).values
        GAPS.append(z[:, top - 1] - z[:, top])
    out = []
    for t in range(h.shape[0]):
        y = torch.zeros_like(h[t])
        for e in torch.argsort(scores[t], descending=True, stable=True)[:top].tolist():
            x = scores[t, e] * h[t]
            y = y + w[f"{p}e{e}.down"] @ _r(square_of_relu(w[f"{p}e{e}.up"] @ x))
        out.append(y)
    return torch.stack(out)


# ---------------------------------------------------------------------------- the model
class Plain:
    """One sequence: `run` takes its next tokens and returns their logits [T, vocab]."""

    def __init__(self, cfg, w):
        self.cfg, self.w = cfg, w
        self.st = [dict() for _ in cfg["layers"]]

    def run(self, tokens, after_layers=None):
        cfg, w, eps = self.cfg, self.w, self.cfg["norm"]["eps"]
        x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
        for i, l in enumerate(cfg["layers"]):
            p, m, f, st = f"l{i}.", l["mixer"], l.get("mlp"), self.st[i]
            h = _r(rms(x, eps) * (1 + w[p + "norm1"]))
            y = {"attention": attention, "parallel": side_by_side}[l["type"]](h, w, p + "mix.", m, eps, st)
            if f:
                y = y + (dense_ff(h, w, p + "mlp.") if f["kind"] == "dense" else experts_ff(h, w, p + "mlp.", f))
            x = x + y
            if after_layers is not None:
                after_layers.append(x.clone())
        return _r(rms(x, eps) * (1 + w["final.norm"])) @ w["embed"].t() * cfg.get("logit_scale", 1.0)


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
