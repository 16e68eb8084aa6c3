"""Kasarax on the GPU against the plain implementation (tests/plain_kasarax.py): each mechanism alone (the query/key/value preparation
with every option, attention behind short convolutions, attention with biases, a query temperature and one added to the denominator,
lightning attention, the pair of mixers, experts weighed on their input, the one-norm block with an output bias), then whole models
through the engine's step function in true 32-bit and in bfloat16: whole prompts, prompts followed by token-by-token decoding, portions
down to two tokens, batches of unequal requests, pages and state slots that are given back and used again, attention made sharp so that
a lost key shows, decays so slow that a lost state shows hundreds of tokens later, long decoding, greedy generation through the
scheduler, and replay through bin/trace_run."""
import json

import numpy as np
import pytest
import torch

import llmengine
import plain_kasarax as P
from gpu_helpers import DEV, Harness
from llmengine.config.kasarax import KasaraxConfig
from llmengine.models.kasarax import describe_kasarax
from llmengine.ops import KernelError, get_ops
from llmengine.parts import LayerCache, build_part
from llmengine.parts.registry import part_class
from tiny import MIXED_SIZES_LONG, Trace, random_ids, round64, run_trace, trace_mixed, trace_portions, trace_tail, trace_whole
from tiny_kasarax import KASARAX, KASARAX_A, KASARAX_B, KASARAX_C, att, config, decided_ids, dense, layer, left, make_tensors, moe, pair, right, write_model

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]
NAMES = {torch.float32: "fp32", torch.bfloat16: "bf16"}


def close(got, want, dt, what="", tol32=1e-4, tol16=4e-2):
    """float32: element by element; bfloat16: the root mean square of the difference against that of the values."""
    got, want = np.asarray(got, dtype=np.float64), np.asarray(want, dtype=np.float64)
    assert np.isfinite(got).all(), what
    if dt == torch.float32:
        err = np.abs(got - want).max() / max(1.0, np.abs(want).max())
        assert err < tol32, f"{what}: float32 differs by {err:.3e}"
    else:
        err = np.sqrt(((got - want) ** 2).mean()) / max(np.sqrt((want ** 2).mean()), 1e-6)
        assert err < tol16, f"{what}: bfloat16 differs by {err:.3e} of the values' size"


def rounded_forward(pc, pw, ids):
    """The plain implementation with the operands of its matrix products rounded to bfloat16, as a 16-bit engine rounds them:
    its distance from the plain logits is the error that rounding alone causes in this model, on these tokens."""
    P.ROUNDING = lambda x: x.to(torch.bfloat16).to(x.dtype)
    try:
        return P.forward(pc, pw, ids).numpy()
    finally:
        P.ROUNDING = None


def rows_close(got, want, dt, what="", rounded=None):
    """Logits of a request, a row a position. float32: as close(). bfloat16: a row's error is the root mean square of its difference
    against that of all values; every row stays within 4 times the largest, and the median row within 3 times the median, of the
    errors that the plain implementation makes with the same roundings (`rounded`)."""
    if dt == torch.float32:
        return close(got, want, dt, what)
    got, want = np.asarray(got, dtype=np.float64), np.asarray(want, dtype=np.float64)
    size = max(np.sqrt((want ** 2).mean()), 1e-6)
    e = np.sqrt(((got - want) ** 2).mean(1)) / size
    n = np.sqrt(((np.asarray(rounded, dtype=np.float64) - want) ** 2).mean(1)) / size
    assert np.median(e) < 3 * np.median(n) + 5e-3, f"{what}: median row differs by {np.median(e):.3e}; rounding alone: {np.median(n):.3e}"
    assert e.max() < 4 * n.max() + 5e-3, f"{what}: row {e.argmax()} differs by {e.max():.3e}; rounding alone: {n.max():.3e} at most"


def whole(d):
    return d if d.dim() == 2 else d.sum(0)


def one_layer(l, width=80, eps=1e-5):
    return config(64, width, eps, 1.0, [l], 2048)


def layer_tensors(cfg, i, dt, sharp=False, seed=5):
    """The tensors of layer i as the file would hold them -> (float64 for the plain side, on the device as the loader hands them
    over: matrices in the engine's precision, everything else float32, the block's description)."""
    t = {k: v for k, v in make_tensors(cfg, seed, dt, sharp).items() if k.startswith(f"l{i}.")}
    spec = describe_kasarax(KasaraxConfig.from_dict(cfg)).layers[i]
    needs = {n.name: n for n in part_class("block", spec.kind).tensor_needs(spec)}
    assert set(needs) == set(t), "the test's tensors and the description's differ"
    dev = {k: v.to(DEV, dt if needs[k].precision == "compute" else torch.float32) for k, v in t.items()}
    return {k: v.double() for k, v in t.items()}, dev, spec


def cache_for(dt, page, part, pages=160):
    h = Harness(dt, page=page, pages=pages)
    c = LayerCache(group=0)
    for need in part.cache_needs():
        if hasattr(need, "head_dim"):
            c.k = torch.zeros(pages + 1, need.num_kv_heads, page, need.head_dim, dtype=dt, device=DEV)
            c.v = torch.zeros(pages + 1, need.num_kv_heads, page, need.value_dim, dtype=dt, device=DEV)
        else:
            c.states[need.name] = torch.zeros((5,) + tuple(need.shape), dtype=need.dtype, device=DEV)
    return h, c


def loaded(category, dt, spec, dev, page=4, pages=160):
    part = build_part(category, spec, Harness(dt).env)
    h, cache = cache_for(dt, page, part if category == "mixer" else part.mixer, pages)
    part = build_part(category, spec, h.env)
    part.load(dev)
    return part, h, cache


PORTIONS = ((0, 1), (1, 3), (3, 4), (4, 21), (21, 22), (22, 24), (24, 95), (95, 96), (96, 97), (97, 140))


def run_in_portions(part, h, cache, x, plain_step, dt, portions=PORTIONS, **tol):
    for lo, hi in portions:
        got = whole(part.forward(x[lo:hi].to(DEV), h.ctx([(1, hi - lo, [])]), cache)).cpu()
        close(got, plain_step(x[lo:hi].double()), dt, f"positions {lo}..{hi}", **tol)


# ---------------------------------------------------------------------------------------------- mechanisms alone
ROW_CASES = [  # heads, kv_heads, dk, dv, rotated, neighbours, norm, taps, bias, temperature, parts
    (6, 2, 18, 10, 8, True, "wide", 3, None, False, 1), (4, 4, 32, 64, 32, True, "wide", 4, None, False, 3),
    (4, 2, 64, 32, 0, False, None, 0, "qkv", True, 2), (3, 1, 10, 6, 0, True, None, 0, "qkv", True, 1),
    (5, 5, 16, 16, 8, False, "wide", 2, "qk", False, 1), (8, 2, 128, 64, 64, False, "head", 5, "qkv", True, 4),
    (2, 1, 300, 20, 300, True, "head", 1, None, True, 1), (40, 8, 128, 128, 32, True, "wide", 3, None, False, 1), (1, 1, 2, 4, 2, True, None, 16, "qk", True, 2)]


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("case", ROW_CASES, ids=[str(c[0]) + "x" + str(c[2]) + "-" + str(c[6]) + "-" + str(c[7]) for c in ROW_CASES])
def test_query_key_value_preparation_alone(dt, case):
    """From a product's sums (in one part and in several) through convolution, biases, norms, rotation and temperature into the
    queries and the pages, for portions of three requests side by side, single tokens (which renew the slots in the same kernel) and
    long portions (whose rows are read by the next ones), a slot used again; what lies beside the columns stays unread."""
    H, G, dk, dv, rot, neighbours, norm, taps, bias_of, temp, n_parts = case
    g = torch.Generator().manual_seed(H + dk + taps)
    nq, nk, nv = H * dk, G * dk, G * dv
    C, extra, T, eps = nq + nk + nv, 8 if (nq + nk + nv) % 4 == 0 else 3, 700, 1e-5
    ids = (1, 2, 3, 4)
    sums = {r: torch.randn(n_parts, T, C + extra, generator=g) / n_parts ** 0.5 for r in ids}
    conv = torch.randn(taps, C, generator=g) if taps else None
    bias = {None: None, "qk": torch.randn(nq + nk, generator=g), "qkv": torch.randn(C, generator=g)}[bias_of]
    wq = wk = None
    if norm:
        wq, wk = (1.0 + 0.3 * torch.randn(n if norm == "wide" else dk, generator=g) for n in (nq, nk))
    inv_f = torch.tensor([50.0 ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=torch.float64) if rot else None
    ang = torch.arange(T, dtype=torch.float64)[:, None] * inv_f[None] if rot else None
    cos, sin = (ang.cos().float().to(DEV), ang.sin().float().to(DEV)) if rot else (None, None)
    mul = (1.0 + 0.3 * torch.log(1.0 + torch.arange(T, dtype=torch.float64) // 5)).float() if temp else None

    def plain(r, pos):
        rows = sums[r].double().sum(0)[:, :C]
        x = rows[pos]
        if taps:
            x = sum(conv[j].double() * rows[pos - (taps - 1) + j] for j in range(taps) if pos - (taps - 1) + j >= 0)
        if bias is not None:
            x = x.clone()
            x[:bias.numel()] += bias.double()
        out = []
        for lo, heads, w in ((0, H, wq), (nq, G, wk)):
            y = x[lo:lo + heads * dk].view(heads, dk).clone()
            if norm == "wide":
                y = (P.rms(y.reshape(-1), eps) * w.double()).view(heads, dk)
            elif norm == "head":
                y = P.rms(y, eps) * w.double()
            if rot and neighbours:
                y = P.rotate_neighbours(y, pos, {"dims": rot, "base": 50.0})
            elif rot:
                c, s, h2 = ang[pos].cos(), ang[pos].sin(), rot // 2
                u, v = y[:, :h2].clone(), y[:, h2:rot].clone()
                y[:, :h2], y[:, h2:rot] = u * c - v * s, v * c + u * s
            out.append(y)
        return out[0] * (float(mul[pos]) if temp else 1.0), out[1], x[nq + nk:].view(G, dv)

    page, pages = 8, 4 * (T // 8 + 2)
    h = Harness(dt, page=page, pages=pages, slots=3)
    kc, vc = (torch.full((pages + 1, G, page, d), 7.0, dtype=dt, device=DEV) for d in (dk, dv))
    state = torch.zeros(4, taps - 1, C, device=DEV) if taps > 1 else None
    devs = [None if t is None else t.to(DEV) for t in (wq, wk, bias, conv, mul)]
    at = {r: 0 for r in ids}
    for batch, end in (([(1, 3), (2, 5)], []), ([(1, 1), (2, 1)], []), ([(1, 1), (2, 70), (3, 2)], [2]), ([(1, 1), (3, 1)], []), ([(3, 9), (4, 1)], []),
                       ([(1, 1), (3, 1), (4, 1)], []), ([(4, 560), (1, 2)], [])):
        ctx = h.ctx([(r, n, []) for r, n in batch])
        if state is not None:
            for i, (r, n) in enumerate(batch):
                if at[r] == 0:
                    state[int(ctx.seq_slot[i])] = 0.0
        rows = torch.cat([sums[r][:, at[r]:at[r] + n] for r, n in batch], dim=1).contiguous().to(DEV)
        q = torch.empty(rows.shape[1], nq, dtype=dt, device=DEV)
        get_ops().qkv_prep(rows, H, G, dk, dv, devs[0], devs[1], eps, cos, sin, ctx, ctx.block_tables[0], q, kc, vc, norm_wide=norm == "wide",
                           bias=devs[2], neighbours=neighbours, conv=devs[3], conv_state=state, q_mul=devs[4])
        row = 0
        for i, (r, n) in enumerate(batch):
            for pos in range(at[r], at[r] + n):
                if n < 100 or pos % 37 == 0 or pos - at[r] < 20:
                    pq, pk, pv = plain(r, pos)
                    pg = int(ctx.block_tables[0][i, pos // page])
                    for got, want, what in ((q[row].float().cpu().view(H, dk), pq, "q"), (kc[pg, :, pos % page].float().cpu(), pk, "k"),
                                            (vc[pg, :, pos % page].float().cpu(), pv, "v")):
                        close(got, want, dt, f"{what} of request {r} at {pos}", tol32=2e-5, tol16=4e-3)
                row += 1
            at[r] += n
        for r in end:
            h.cm.release(r)
    assert (kc[pages] == 7.0).all()


def test_preparation_refuses_what_it_cannot_do():
    h = Harness(torch.float32)
    ctx = h.ctx([(1, 2, [])])
    parts, q = torch.zeros(1, 2, 4 * 8, device=DEV), torch.zeros(2, 16, device=DEV)
    args = (parts, 2, 1, 8, 8, None, None, 1e-5, None, None, ctx, ctx.block_tables[0], q, None, None)
    with pytest.raises(KernelError):
        get_ops().qkv_prep(*args, q_mul=torch.ones(9, device=DEV), unit_rms=True)
    with pytest.raises(KernelError):
        get_ops().qkv_prep(*args, conv=torch.ones(17, 32, device=DEV), conv_state=torch.zeros(5, 16, 32, device=DEV))


def _conv_attention(heads, kv_heads, dim, vdim, conv, rot):
    return one_layer(pair(left(heads, kv_heads, dim, vdim, dim ** -0.5, conv, rot), right(1, 4, 4, (0.5,))))


LEFT_CASES = [(KASARAX_A, 1), (KASARAX_A, 2), (KASARAX_B, 0), (KASARAX_B, 1), (KASARAX_B, 4), (KASARAX_C, 0), (KASARAX_C, 2),
              (_conv_attention(8, 1, 128, 128, 4, (64, 5e5)), 0), (_conv_attention(2, 2, 96, 40, 6, (24, 1e4)), 0), (_conv_attention(2, 1, 300, 20, 2, (2, 9.0)), 0)]


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("cfg,i", LEFT_CASES, ids=["a1", "a2", "b0", "b1", "b4", "c0", "c2", "128", "96", "300"])
@pytest.mark.parametrize("sharp", [False, True])
def test_attention_behind_convolutions_alone(dt, cfg, i, sharp):
    """Over a prompt portion, then over single tokens and further portions that read the first one's cache rows and convolution inputs;
    one to six taps; rotation of a part of a head, all of it and none; head sizes of every attention kernel, keys and values of
    different sizes."""
    cpu, dev, spec = layer_tensors(cfg, i, dt, sharp)
    part, h, cache = loaded("mixer", dt, spec.mixer.left, dev)
    m, state = cfg["layers"][i]["mixer"]["left"], {}
    x = torch.randn(140, cfg["width"], generator=torch.Generator().manual_seed(6)).to(dt)
    run_in_portions(part, h, cache, x, lambda xs: P.conv_attention(xs, cpu, f"l{i}.mix.left.", m, cfg["norm"]["eps"], state), dt, tol16=6e-2 if sharp else 4e-2)


def _attention(heads, kv_heads, dim, vdim, temp):
    return one_layer(layer("attention", att(heads, kv_heads, dim, vdim, dim ** -0.5, temp)))


ATTENTION_CASES = [(KASARAX_A, 0), (KASARAX_A, 3), (KASARAX_B, 2), (KASARAX_B, 3), (KASARAX_C, 1), (KASARAX_C, 3), (_attention(8, 1, 128, 32, (0.5, 20)), 0),
                   (_attention(6, 2, 96, 128, (0.2, 3)), 0), (_attention(2, 1, 300, 16, None), 0)]


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("cfg,i", ATTENTION_CASES, ids=["a0", "a3", "b2", "b3", "c1", "c3", "128", "96", "300"])
@pytest.mark.parametrize("sharp", [False, True])
def test_attention_with_biases_and_a_query_temperature_alone(dt, cfg, i, sharp):
    cpu, dev, spec = layer_tensors(cfg, i, dt, sharp)
    part, h, cache = loaded("mixer", dt, spec.mixer, dev)
    m, state = cfg["layers"][i]["mixer"], {}
    x = torch.randn(140, cfg["width"], generator=torch.Generator().manual_seed(8)).to(dt)
    run_in_portions(part, h, cache, x, lambda xs: P.attention(xs, cpu, f"l{i}.mix.", m, cfg["norm"]["eps"], state), dt, tol16=6e-2 if sharp else 4e-2)


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("sink", [-40.0, 0.0, 12.0])
def test_sink_alone(dt, sink):
    """A sink that nothing notices, one that counts as a key with a score of zero, one that takes nearly all the weight; a first
    token (whose only other term is its own) in a prompt and decoded."""
    cfg = one_layer(pair(left(4, 2, 32, 64, 0.2, 2, (8, 100.0)), right(1, 4, 4, (0.5,))))
    cpu, dev, spec = layer_tensors(cfg, 0, dt)
    cpu["l0.mix.left.sink"] = torch.full((4,), sink, dtype=torch.float64)
    dev["l0.mix.left.sink"] = torch.full((4,), sink, device=DEV)
    part, h, cache = loaded("mixer", dt, spec.mixer.left, dev)
    state = {}
    x = torch.randn(30, cfg["width"], generator=torch.Generator().manual_seed(9)).to(dt)
    run_in_portions(part, h, cache, x, lambda xs: P.conv_attention(xs, cpu, "l0.mix.left.", cfg["layers"][0]["mixer"]["left"], 1e-5, state), dt,
                    ((0, 1), (1, 2), (2, 20), (20, 21), (21, 30)))


@pytest.mark.parametrize("dt", DTYPES)
def test_one_added_to_the_denominator(dt):
    """Keys whose scores are far below, at and far above zero: what the added one takes goes from nearly all of the weight to none, and
    the scores that nobody reaches (all of them -60) give a result near zero, not their mean."""
    cfg = one_layer(layer("attention", att(2, 2, 32, 32, 1.0)))
    cpu, dev, spec = layer_tensors(cfg, 0, dt)
    q = "l0.mix."
    for name, w in ((q + "q", torch.zeros(64, 80)), (q + "k", torch.zeros(64, 80))):
        cpu[name], dev[name] = w.double(), w.to(DEV, dt)
    for score in (-60.0, -3.0, 0.0, 5.0, 60.0):
        a, b = torch.zeros(64), torch.zeros(64)
        a[0::32], b[0::32] = score, 1.0
        for name, w in ((q + "q.b", a), (q + "k.b", b)):
            cpu[name], dev[name] = w.double(), w.to(DEV)
        part, h, cache = loaded("mixer", dt, spec.mixer, dev)
        state = {}
        x = torch.randn(50, 80, generator=torch.Generator().manual_seed(1)).to(dt)
        run_in_portions(part, h, cache, x, lambda xs: P.attention(xs, cpu, q, cfg["layers"][0]["mixer"], 1e-5, state), dt,
                        ((0, 1), (1, 2), (2, 40), (40, 41), (41, 50)))


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("page", [4, 16])
@pytest.mark.parametrize("decoded", [False, True])
@pytest.mark.parametrize("kind", ["attention", "left"])
def test_a_marked_key_far_back_and_at_page_borders(dt, page, decoded, kind):
    """Hundreds of tokens of which one is marked; later tokens ask for it with a score that stands far out, from right behind it, from
    the next page and from hundreds of tokens away, in the same portion and decoded one by one. Without the marked token the plain
    result is a different one."""
    T, width = 420, 80
    m = att(4, 2, 32, 64, 1.0) if kind == "attention" else left(4, 2, 32, 64, 1.0, 3)
    cfg = one_layer(layer("attention", m) if kind == "attention" else pair(m, right(1, 4, 4, (0.5,))), width)
    p = "l0.mix." if kind == "attention" else "l0.mix.left."
    cpu, dev, spec = layer_tensors(cfg, 0, dt)
    q, k = torch.zeros(128, width), torch.zeros(64, width)
    q[0::32, 0], k[0::32, 1] = 8.0, 8.0                     # the query's first number asks, the key's answers
    new = {"q": q, "k": k}
    if kind == "attention":
        new.update({"q.b": torch.zeros(128), "k.b": torch.zeros(64)})
    else:                                                    # convolutions that let the token itself through; norms that spread scores
        only = torch.zeros(128, 3)
        only[:, 2] = 1.0
        q[1::32, 2], k[2::32, 2] = 1.0, 1.0                  # something that is always there, in directions that never meet
        new.update({"q.conv": only, "k.conv": only[:64], "q.norm": torch.ones(128), "k.norm": torch.ones(64), "sink": torch.zeros(4)})
    for s, w in new.items():
        cpu[p + s], dev[p + s] = w.to(dt).double(), w.to(DEV, dev[p + s].dtype)
    part, h, cache = loaded("mixer", dt, spec.mixer if kind == "attention" else spec.mixer.left, dev, page=page, pages=T // page + 4)
    run = P.attention if kind == "attention" else P.conv_attention
    for marked in (page * 5 - 1, page * 5, 77):
        x = torch.randn(T, width, generator=torch.Generator().manual_seed(marked))
        x[:, :2] = 0
        x[:, 2] = 1.0
        x[marked, 1] = 1.0                       # the key that is looked for
        x[marked, 3:] *= 3.0                     # and what it carries
        asks = [marked + 1, marked + page, marked + 150, T - 1]
        x[asks, 0] = 1.0
        x = x.to(dt)
        want = run(x.double(), cpu, p, m, 1e-5, {})
        cut = marked + 1 if decoded else T
        steps = [(0, cut)] + ([(t, t + 1) for t in range(cut, T)] if decoded else [])
        got = torch.cat([whole(part.forward(x[lo:hi].to(DEV), h.ctx([(marked + 1, hi - lo, [])]), cache)).cpu() for lo, hi in steps])
        close(got, want, dt, f"marked key at {marked}")
        close(got[asks], want[asks], dt, f"asking for {marked}", tol16=2e-2)
        h.cm.release(marked + 1)
        for name in cache.states:
            cache.states[name].zero_()
        x2 = x.double().clone()
        x2[marked, 1] = 0.0
        other = run(x2, cpu, p, m, 1e-5, {})
        assert float((other[asks] - want[asks]).norm()) > 0.5 * float(want[asks].norm()), "the case is meant to depend on the marked key"


def _lightning(heads, dim, vdim):
    return one_layer(pair(left(1, 1, 4, 4, 0.5, 1), right(heads, dim, vdim, [1.0 - 2.0 ** (-1 - i) for i in range(heads)])))


RIGHT_CASES = [(KASARAX_A, 1), (KASARAX_A, 2), (KASARAX_B, 0), (KASARAX_B, 1), (KASARAX_C, 0), (KASARAX_C, 2), (_lightning(8, 128, 128), 0), (_lightning(3, 100, 36), 0),
               (_lightning(5, 16, 130), 0)]


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("cfg,i", RIGHT_CASES, ids=["a1", "a2", "b0", "b1", "c0", "c2", "8x128", "100x36", "16x130"])
def test_lightning_attention_alone(dt, cfg, i):
    """Portions of 1, 2 and many tokens that hand the state on through the slot (activated in the state's kernel and ahead of it);
    decays of 0 and 1 among them; rows of the common norm shorter and longer than a warp takes."""
    cpu, dev, spec = layer_tensors(cfg, i, dt)
    part, h, cache = loaded("mixer", dt, spec.mixer.right, dev)
    m, state = cfg["layers"][i]["mixer"]["right"], {}
    x = torch.randn(140, cfg["width"], generator=torch.Generator().manual_seed(16)).to(dt)
    run_in_portions(part, h, cache, x, lambda xs: P.lightning(xs, cpu, f"l{i}.mix.right.", m, cfg["norm"]["eps"], state), dt)


@pytest.mark.parametrize("dt", DTYPES)
def test_a_state_written_once_is_read_hundreds_of_tokens_later(dt):
    """A decay of one, one token that writes and one that asks along the same direction 400 tokens later, after portions and single
    tokens: a state that is lost, reset or read from another slot on the way shows."""
    cfg = one_layer(pair(left(1, 1, 4, 4, 0.5, 1), right(2, 32, 48, (1.0, 0.99999))))
    cpu, dev, spec = layer_tensors(cfg, 0, dt)
    p = "l0.mix.right."
    q, k = torch.zeros(64, 80), torch.zeros(64, 80)
    q[:, 0], k[:, 1] = 6.0, 6.0
    q[1::2], k[1::2] = 0.0, 0.0
    for s, w in (("q", q), ("k", k)):
        cpu[p + s], dev[p + s] = w.double(), w.to(DEV, dt)
    part, h, cache = loaded("mixer", dt, spec.mixer.right, dev)
    m, T = cfg["layers"][0]["mixer"]["right"], 430
    x = torch.randn(T, 80, generator=torch.Generator().manual_seed(3))
    x[:, :2] = 0.0                                          # silu(0): nothing is written, nothing is asked
    x[3, 1] = 1.0
    x[T - 2, 0] = 1.0
    x = x.to(dt)
    want = P.lightning(x.double(), cpu, p, m, 1e-5, {})
    got, lo = [], 0
    for n in (2, 1, 1, 130, 1, 2, 200, 61, 1, 1, 30):
        got.append(whole(part.forward(x[lo:lo + n].to(DEV), h.ctx([(1, n, [])]), cache)).cpu())
        lo += n
    assert lo == T
    close(torch.cat(got), want, dt, "portions", tol32=2e-4)
    fresh = P.lightning(x[10:].double(), cpu, p, m, 1e-5, {})
    assert float((fresh[T - 12] - want[T - 2]).norm()) > 0.9 * float(want[T - 2].norm()), "the case is meant to depend on token 3"


@pytest.mark.parametrize("dt", DTYPES)
def test_pairs_of_mixers_for_requests_side_by_side(dt):
    """Portions of three requests in one step, short ones and long ones, single tokens among them, each against itself alone: keys and
    values, convolution inputs and the state matrix of a layer at once."""
    cfg, i = KASARAX_B, 0
    cpu, dev, spec = layer_tensors(cfg, i, dt)
    part, h, cache = loaded("mixer", dt, spec.mixer, dev, page=16)
    m, g = cfg["layers"][i]["mixer"], torch.Generator().manual_seed(2)
    x = {r: torch.randn(120, cfg["width"], generator=g).to(dt) for r in (1, 2, 3)}
    st, at = {r: {} for r in x}, {r: 0 for r in x}
    for batch in ([(1, 3), (2, 70), (3, 2)], [(3, 41), (1, 2), (2, 1)], [(2, 1), (3, 1), (1, 1)], [(1, 1), (2, 1)], [(1, 65), (2, 9), (3, 30)]):
        xs = torch.cat([x[r][at[r]:at[r] + n] for r, n in batch])
        got = whole(part.forward(xs.to(DEV), h.ctx([(r, n, []) for r, n in batch]), cache)).cpu()
        lo = 0
        for r, n in batch:
            want = P.side_by_side(x[r][at[r]:at[r] + n].double(), cpu, f"l{i}.mix.", m, 1e-6, st[r])
            close(got[lo:lo + n], want, dt, f"request {r} from {at[r]}")
            lo, at[r] = lo + n, at[r] + n


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("width,ff,experts,top,n", [(128, 96, 6, 1, 5), (128, 96, 6, 1, 300), (128, 64, 4, 3, 70), (70, 22, 5, 2, 33), (96, 40, 3, 3, 9), (64, 128, 2, 1, 700)])
def test_experts_weighed_on_their_input(dt, width, ff, experts, top, n):
    """Few rows an expert and many (every tile of the products), one chosen expert (no sum behind it) and several, all of them; scores from nearly
    0 to nearly 1, so that a weight on the output instead of the input, or a missing one, shows."""
    cfg = one_layer(layer("attention", att(1, 1, 4, 4, 0.5), moe(ff, experts, top)), width)
    cpu, dev, spec = layer_tensors(cfg, 0, dt)
    part = build_part("feed_forward", spec.feed_forward, Harness(dt).env)
    part.load(dev)
    x = torch.randn(n, width, generator=torch.Generator().manual_seed(n)).to(dt)
    if n > 100:
        x[:40] = x[0] * 1.001  # an expert with many rows
    h = Harness(dt, pages=400)
    got = whole(part.forward(x.to(DEV), h.ctx([(1, n, [])]))).cpu()
    want = P.experts_ff(x.double(), cpu, "l0.mlp.", cfg["layers"][0]["mlp"])
    scores = torch.sort(P.sigmoid(x.double() @ cpu["l0.mlp.router"].t()), dim=1, descending=True).values
    sure = torch.ones(n, dtype=torch.bool) if top == experts else scores[:, top - 1] - scores[:, top] > 1e-4   # (not a tie within rounding)
    assert int(sure.sum()) > 0.9 * n
    close(got[sure], want[sure], dt, "experts", tol16=2e-2)
    some = slice(n - min(n, 20), n)                           # the weights on the outputs: a different result
    out = torch.zeros_like(want)
    s = P.sigmoid(x.double() @ cpu["l0.mlp.router"].t())
    for t in range(n)[some]:
        for e in torch.argsort(s[t], descending=True, stable=True)[:top].tolist():
            out[t] += s[t, e] * (cpu[f"l0.mlp.e{e}.down"] @ P.square_of_relu(cpu[f"l0.mlp.e{e}.up"] @ x[t].double()))
    assert float((out[some] - want[some]).norm()) > 0.05 * float(want[some].norm())


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("heads,dv,act", [(1, 2048, "sigmoid"), (1, 513, "silu"), (3, 700, "sigmoid"), (1, 512, "sigmoid")])
def test_norm_and_gate_of_wide_rows(dt, heads, dv, act):
    g = torch.Generator().manual_seed(dv)
    n, parts, off = 37, 3, 5
    o, w, gate = torch.randn(n, heads * dv, generator=g), 1 + 0.3 * torch.randn(heads * dv, generator=g), torch.randn(parts, n, heads * dv + off + 2, generator=g)
    out = torch.empty(n, heads * dv, dtype=dt, device=DEV)
    get_ops().head_norm_gate(o.to(DEV), w.to(DEV), gate.to(DEV), off, 1e-5, out, n, heads, dv, act=act)
    z = gate.double().sum(0)[:, off:off + heads * dv]
    want = (P.rms(o.double().view(n, heads, dv), 1e-5).reshape(n, -1) * w.double()) * (P.sigmoid(z) if act == "sigmoid" else P.silu(z))
    close(out.float().cpu(), want, dt, tol32=1e-5, tol16=5e-3)


@pytest.mark.parametrize("parts,width,off,cols", [(1, 64, 8, 40), (3, 61, 5, 33), (2, 128, 0, 128)])
def test_activated_sums(parts, width, off, cols):
    x = torch.randn(parts, 29, width, generator=torch.Generator().manual_seed(cols)) * 3
    out = torch.empty(29, cols, device=DEV)
    get_ops().silu_sums(x.to(DEV), off, cols, out, 29)
    close(out.cpu(), P.silu(x.double().sum(0)[:, off:off + cols]), torch.float32, tol32=1e-6)


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("cfg,i", [(KASARAX_A, 0), (KASARAX_A, 1), (KASARAX_A, 2), (KASARAX_B, 0), (KASARAX_B, 1), (KASARAX_B, 2), (KASARAX_B, 3), (KASARAX_C, 1),
                                   (KASARAX_C, 3)], ids=["a0", "a1", "a2", "b0", "b1", "b2", "b3", "c1", "c3"])
def test_block_alone(dt, cfg, i):
    """A whole layer on a float32 stream: one norm (weight 1 + w) for both sub-layers; with a feed-forward the output projection's bias is
    added where both results enter the stream, without one by the mixer."""
    from llmengine.parts.base import Residual
    cpu, dev, spec = layer_tensors(cfg, i, dt)
    block, h, cache = loaded("block", dt, spec, dev)
    eps, l, p = cfg["norm"]["eps"], cfg["layers"][i], f"l{i}."
    f = cfg["layers"][i]["mlp"]
    x = torch.randn(240, cfg["width"], generator=torch.Generator().manual_seed(46)) + 0.5
    if f and f["kind"] == "moe" and f["router"]["top"] < f["router"]["experts"]:  # rows on which the router has no close call
        z = (P.rms(x.double(), eps) * (1 + cpu[p + "norm1"])) @ cpu[p + "mlp.router"].t()
        z = torch.sort(z, dim=1, descending=True).values
        x = x[z[:, f["router"]["top"] - 1] - z[:, f["router"]["top"]] > 0.1]
    x = x[:60]
    assert x.shape[0] == 60
    state, lo = {}, 0
    mix = {"attention": P.attention, "parallel": P.side_by_side}[l["type"]]
    for n in (17, 1, 2, 40):
        want = x[lo:lo + n].double()
        hh = P.rms(want, eps) * (1 + cpu[p + "norm1"])
        want = want + mix(hh, cpu, p + "mix.", l["mixer"], eps, state)
        if f:
            want = want + (P.dense_ff(hh, cpu, p + "mlp.") if f["kind"] == "dense" else P.experts_ff(hh, cpu, p + "mlp.", f))
        res = block.forward(Residual(x[lo:lo + n].to(DEV).contiguous()), h.ctx([(1, n, [])]), cache)
        if res.pending is not None:
            get_ops().residual_add(res.h, res.pending)
        close(res.h.float().cpu(), want, dt, f"tokens {lo}..{lo + n}", tol32=3e-4, tol16=6e-2)
        lo += n


# ---------------------------------------------------------------------------------------------- whole models
def replay(eng, trace):
    """The trace's steps through Engine.run_step, in this process -> {(request, position): logits row}."""
    ids, nxt, out = {}, 1, {}
    for k, s in enumerate(trace.steps):
        batch = []
        for e in s["entries"]:
            if e["id"] not in ids:
                ids[e["id"]], nxt = nxt, nxt + 1
            batch.append((ids[e["id"]], e["tokens"], e["want"]))
        lg = eng.run_step(batch, end=[ids[n] for n in s["end"]]).float().cpu().numpy()
        for n in s["end"]:
            ids.pop(n)
        for i, key in enumerate(trace.rows.get(k, [])):
            out[key] = lg[i].copy()
    return out


@pytest.fixture(scope="module", params=[(n, dt, sharp) for n in ("ka", "kb", "kc") for dt in DTYPES for sharp in (False, True)
                                        if not (sharp and n == "kc")],
                ids=lambda p: f"{p[0]}-{NAMES[p[1]]}{'-sharp' if p[2] else ''}")
def model(request, tmp_path_factory):
    name, dt, sharp = request.param
    cfg, page = KASARAX[name]
    d = write_model(str(tmp_path_factory.mktemp("kasarax")), cfg, dt, sharp=sharp)
    pc, pw = P.read_model(d)
    lens = [5, 64, 33, 130, 97] if name != "kb" else [3, 47, 64, 200, 129]
    reqs = {f"r{i}": decided_ids(pc, pw, n, 50 + i) for i, n in enumerate(lens)}  # (no router within rounding of another choice)
    plain = {k: P.forward(pc, pw, v).numpy() for k, v in reqs.items()}
    if dt == torch.bfloat16:
        plain.update({k + ".rounded": rounded_forward(pc, pw, v) for k, v in reqs.items()})
    eng = llmengine.Engine(d, NAMES[dt], block_size=page)
    longest = max(round64(len(v)) for v in reqs.values())
    tokens = longest + 3 * 64  # room for the longest request and three short ones: pages are used again
    eng.configure_cache(num_blocks=tokens // page, block_size=page, num_slots=4)
    return dt, eng, reqs, plain, tokens, (pc, pw), cfg


@pytest.mark.parametrize("cut", ["whole", "tail", "portions", "mixed"])
def test_cuts_match_plain_and_one_another(model, cut):
    """whole: each prompt in one step; tail: its last 32 tokens one by one (prefill against decoding through the cache and the
    state); portions: sizes 7, 2, 13, 2, 5, 3, ... ; mixed: up to four live requests, portions beside single tokens, with so few
    pages and slots that both are used again."""
    dt, eng, reqs, plain, tokens, _, _ = model
    named = {f"{cut}.{k}": v for k, v in reqs.items()}
    trace = {"whole": trace_whole, "tail": trace_tail, "portions": trace_portions}[cut](named) if cut != "mixed" else \
        trace_mixed(named, tokens, seed=5, sizes=MIXED_SIZES_LONG)
    rows = replay(eng, trace)
    assert eng.cm.num_requests == 0
    for k, ids in reqs.items():
        got = np.stack([rows[(f"{cut}.{k}", p)] for p in range(len(ids))])
        rows_close(got, plain[k], dt, f"{cut}, request {k}", plain.get(k + ".rounded"))


def test_the_stream_after_every_layer(model):
    """In float32 the residual stream behind every layer against the plain one."""
    dt, eng, reqs, _, _, (pc, pw), cfg = model
    if dt != torch.float32:
        pytest.skip("compared in float32")
    ids = reqs["r2"]
    after, got = [], []
    P.forward(pc, pw, ids, after_layers=after)
    m = eng._ensure_model()
    m.after_run = lambda r, h: got.append(h[:len(ids)].float().cpu().clone())
    try:
        eng.run_step([(9, ids, [len(ids) - 1])], end=[9])
    finally:
        m.after_run = None
    assert len(got) == len(after) == len(cfg["layers"])
    for r, (a, b) in enumerate(zip(got, after)):
        close(a, b, dt, f"layer {r}")


def test_keys_at_page_borders_and_first_tokens(model):
    """A request that grows one token a step from its first token across page borders, beside a second one that starts later (so that
    its pages lie between the first one's, and its state in another slot)."""
    dt, eng, reqs, plain, _, _, _ = model
    a, b = reqs["r2"], reqs["r1"][:20]
    t = Trace()
    for p in range(len(a)):
        entries = [("a", a[p:p + 1], [0], p)]
        if 5 <= p < 5 + len(b):
            entries.append(("b", b[p - 5:p - 4], [0], p - 5))
        t.add(entries, end=[n for n, cond in (("a", p == len(a) - 1), ("b", p == 4 + len(b))) if cond])
    rows = replay(eng, t)
    rows_close(np.stack([rows[("a", p)] for p in range(len(a))]), plain["r2"], dt, "token by token", plain.get("r2.rounded"))
    rows_close(np.stack([rows[("b", p)] for p in range(len(b))]), plain["r1"][:20], dt, "the request beside it",
               plain["r1.rounded"][:20] if dt == torch.bfloat16 else None)


def test_a_batch_of_unequal_requests_against_each_alone(model):
    """Four requests of unequal length in ONE step, then each alone: the same rows (float32: to rounding)."""
    dt, eng, reqs, plain, _, _, _ = model
    names = ["r0", "r2", "r1", "r4"]
    lg = eng.run_step([(20 + i, reqs[k], list(range(len(reqs[k])))) for i, k in enumerate(names)], end=[20, 21, 22, 23]).float().cpu().numpy().copy()
    lo = 0
    for k in names:
        n = len(reqs[k])
        alone = eng.run_step([(30, reqs[k], list(range(n)))], end=[30]).float().cpu().numpy()
        rows_close(lg[lo:lo + n], plain[k], dt, f"{k} in the batch", plain.get(k + ".rounded"))
        if dt == torch.float32:
            close(lg[lo:lo + n], alone, dt, f"{k}: batch against alone", tol32=2e-5)
        else:
            rows_close(lg[lo:lo + n], alone, dt, f"{k}: batch against alone", plain[k + ".rounded"] - plain[k] + alone)
        lo += n


def test_a_slot_that_is_used_again_starts_at_zero(model):
    """Requests one after the other in an engine with a single live request at a time: each gets the one before's slot and pages,
    and must not see its state, its convolution inputs or its keys."""
    dt, eng, reqs, plain, _, _, _ = model
    for k in ("r3", "r1", "r3"):
        n = len(reqs[k])
        got = eng.run_step([(77, reqs[k], list(range(n)))], end=[77]).float().cpu().numpy()
        rows_close(got, plain[k], dt, k, plain.get(k + ".rounded"))


def test_long_decoding_and_generation(model):
    """Greedy generation through the engine's entry point and scheduler (decode steps replay CUDA graphs in bfloat16); in
    float32 the tokens are the plain implementation's."""
    dt, eng, reqs, plain, _, (pc, pw), cfg = model
    prompt = reqs["r2"][:11]
    out, reason = eng.generate(prompt, 90)
    assert reason == "length" and len(out) == 101 and out[:11] == prompt
    logits = P.forward(pc, pw, out).numpy()
    slack = 1e-4 if dt == torch.float32 else 0.1
    if dt == torch.bfloat16:  # (rows that rounding alone moves far, at a router's close call say, may choose another token)
        slack = max(slack, 3 * float(np.abs(rounded_forward(pc, pw, out) - logits).max()) / max(1.0, float(np.abs(logits).max())))
    for p in range(10, 100):  # the chosen token is the plain logits' best, or ties with it within rounding
        assert logits[p, out[p + 1]] >= logits[p].max() - slack * max(1.0, np.abs(logits[p]).max()), p


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("dim,vdim,conv", [(64, 32, 4), (32, 128, 3), (128, 64, 2), (48, 40, 3)])
def test_single_tokens_behind_long_contexts(dt, dim, vdim, conv, tmp_path):
    """Three requests of unequal length (up to 1,000 tokens) whose last tokens come one a step, side by side: single tokens whose
    key range is cut into pieces that run side by side and are merged, keys and values of different sizes, a learned sink and the added
    one where the pieces are merged, a gate a head behind them; a state and convolution inputs carried through it all."""
    layers = [layer("attention", att(4, 2, dim, vdim, 1.0 / dim ** 0.5, (0.3, 100)), dense(64)),
              pair(left(4, 2, dim, vdim, 1.0 / dim ** 0.5, conv, (dim // 2, 1e4)), right(2, 32, 48, (0.9, 0.9995)), dense(48)),
              layer("attention", att(3, 1, vdim, dim, 1.0 / vdim ** 0.5))]
    cfg = config(120, 64, 1e-5, 0.7, layers, 2048)
    d = write_model(str(tmp_path / "m"), cfg, dt, sharp=True)
    pc, pw = P.read_model(d)
    reqs = {"a": random_ids(1000, 120, 1), "b": random_ids(500, 120, 2), "c": random_ids(120, 120, 3)}
    tail = 12
    eng = llmengine.Engine(d, NAMES[dt], block_size=16)
    eng.configure_cache(num_blocks=(1024 + 512 + 128) // 16, block_size=16, num_slots=4)
    ids = {"a": 1, "b": 2, "c": 3}
    for k, v in reqs.items():
        eng.run_step([(ids[k], v[:-tail], [])], end=[])
    rows = {k: [] for k in reqs}
    for t in range(tail):
        batch = [(ids[k], [v[len(v) - tail + t]], [0]) for k, v in reqs.items()]
        lg = eng.run_step(batch, end=list(ids.values()) if t == tail - 1 else []).float().cpu().numpy()
        for i, k in enumerate(reqs):
            rows[k].append(lg[i].copy())
    for k, v in reqs.items():
        want = P.forward(pc, pw, v).numpy()[-tail:]
        rounded = rounded_forward(pc, pw, v)[-tail:] if dt == torch.bfloat16 else None
        rows_close(np.stack(rows[k]), want, dt, f"request {k}", rounded)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["ka", "kb"])
def test_replay_through_the_command(dtype, name, tmp_path):
    """bin/trace_run as a user runs it."""
    cfg, page = KASARAX[name]
    dt = torch.float32 if dtype == "float32" else torch.bfloat16
    d = write_model(str(tmp_path / "m"), cfg, dt)
    pc, pw = P.read_model(d)
    reqs = {f"q{i}": decided_ids(pc, pw, n, 80 + i) for i, n in enumerate([2, 70, 35, 150])}
    t = trace_mixed(reqs, 256 + 64, seed=3, sizes=MIXED_SIZES_LONG)
    rows = run_trace(d, dtype, t, str(tmp_path / "out"), 256 + 64, page, cfg["vocab"])
    for k, ids in reqs.items():
        rows_close(np.stack([rows[(k, p)] for p in range(len(ids))]), P.forward(pc, pw, ids).numpy(), dt, k,
                   rounded_forward(pc, pw, ids) if dtype == "bfloat16" else None)


def test_generation_from_the_command_line(tmp_path):
    from test_cli import run_cli
    d = write_model(str(tmp_path / "model"), KASARAX_C, torch.float32)
    r = run_cli("--model", d, "--prompt-ids", "5,17,3,90", "--max-new", "6", "--block-size", "8", "--num-blocks", "32")
    assert r.returncode == 0, r.stderr
    line = [json.loads(l) for l in r.stdout.splitlines() if l.startswith("{")][0]
    pc, pw = P.read_model(d)
    assert line["token_ids"] == P.greedy(pc, pw, [5, 17, 3, 90], 6) and line["finish_reason"] == "length"
