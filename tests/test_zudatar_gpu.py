"""Zudatar on the GPU against the plain implementation (tests/plain_zudatar.py): each mechanism alone (the pair embedding with its
previous token, the delta rule with a decay per key channel and its low-rank maps, attention whose values are its keys, latent
attention with a sink, a window and borrowed latents, the factor on the logits, the block), then whole models through the engine's
step function in true 32-bit and in bfloat16: whole prompts, prompts followed by token-by-token decoding, portions down to two
tokens, batches of unequal requests, pages and state slots that are given back and used again, attention made sharp so that a key
that is lost or let through a window's edge shows, decays so slow that a lost state shows hundreds of tokens later, long decoding,
greedy generation through the scheduler, and replay through bin/trace_run."""
import json

import numpy as np
import pytest
import torch

import llmengine
import plain_zudatar as P
from gpu_helpers import DEV, Harness
from llmengine.config.zudatar import ZudatarConfig
from llmengine.models.zudatar import describe_zudatar
from llmengine.ops import get_ops
from llmengine.parts import LayerCache, build_part
from llmengine.parts.registry import part_class
from tiny import MIXED_SIZES_LONG, Trace, random_ids, round64, run_trace, trace_mixed, trace_portions, trace_tail, trace_whole
from tiny_zudatar import ZUDATAR, ZUDATAR_A, ZUDATAR_B, ZUDATAR_C, att, config, delta, lat, layer, make_tensors, ranks_of, sharpened, write_model

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]
NAMES = {torch.float32: "fp32", torch.bfloat16: "bf16"}


def close(got, want, dt, what="", tol32=1e-4, tol16=4e-2):
    """float32: element by element; bfloat16: the root mean square of the difference against that of the values."""
    got, want = np.asarray(got, dtype=np.float64), np.asarray(want, dtype=np.float64)
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


def one_layer(l, width=80, eps=1e-5, before=()):
    return config(64, width, eps, 2.0, (19, 3, 5), 1.0, list(before) + [l], 2048)


def layer_tensors(cfg, i, dt, sharp=False, seed=5, ranks=None):
    """The tensors of layer i as the file would hold them -> (float64 for the plain side, on the device as the loader hands them
    over: matrices in the engine's precision, everything else float32, the block's description)."""
    ranks = ranks_of(cfg) if ranks is None else ranks
    full = json.loads(json.dumps(cfg))
    for j, l in enumerate(full["layers"]):
        if l["type"] == "channel_delta":
            l["mixer"].update(zip(("decay_rank", "gate_rank"), ranks.get(j, (16, 16))))
    t = {k: v for k, v in make_tensors(cfg, seed, dt, sharp, ranks).items() if k.startswith(f"l{i}.")}
    spec = describe_zudatar(ZudatarConfig.from_dict(full)).layers[i]
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
            if need.value_dim:
                c.v = torch.zeros(pages + 1, need.num_kv_heads, page, need.value_dim, dtype=dt, device=DEV)
            c.window = need.window
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
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("dim,buckets,mp,mc,scale", [(40, 53, 17, 5, 3.7), (1030, 1, 3, 2, 1.0), (128, 769, 2147483647, 2147483640, 0.5), (7, 9, 0, 0, 2.0)])
def test_pair_embedding_alone(dt, dim, buckets, mp, mc, scale):
    """Portions of several requests side by side, single tokens among them, slots used again: every token's row is its own and the
    pair's, the first token of a sequence takes the last row of the table, multipliers far beyond 32 bits when multiplied."""
    from llmengine.parts.spec import EmbeddingSpec
    g = torch.Generator().manual_seed(dim)
    table, pairs = torch.randn(97, dim, generator=g).to(dt), torch.randn(buckets + 1, dim, generator=g).to(dt)
    h = Harness(dt, slots=3)
    spec = EmbeddingSpec("e", 97, dim, kind="lookup_pairs", scale=scale, pair_weight="b", pair_buckets=buckets, pair_mul_prev=mp, pair_mul_cur=mc)
    part = build_part("embedding", spec, h.env)
    part.load({"e": table.to(DEV), "b": pairs.to(DEV)})
    cache = LayerCache()
    cache.states["embedding.previous"] = torch.zeros(4, 1, dtype=torch.int32, device=DEV)
    w = {"embed": table.double(), "bigram": pairs.double()}
    e = {"scale": scale, "bigram": {"buckets": buckets, "mul_prev": mp, "mul_cur": mc}}
    ids = {r: random_ids(40, 97, 60 + r) for r in (1, 2, 3, 4)}
    at, st = {r: 0 for r in ids}, {r: {} for r in ids}
    for batch, end in (([(1, 5)], []), ([(1, 1), (2, 1)], []), ([(2, 2), (1, 2), (3, 7)], [2]), ([(3, 1), (4, 1), (1, 1)], []), ([(4, 30), (1, 9)], [])):
        entries = [(r, ids[r][at[r]:at[r] + n], []) for r, n in batch]
        ctx = h.ctx(entries, vocab=97)
        ctx.embedding_cache = cache
        got = part.forward(ctx).cpu()
        want = torch.cat([P.embedding(toks, w, e, st[r]) for r, toks, _ in entries])
        np.testing.assert_allclose(got.numpy(), want.float().numpy(), rtol=1e-6, atol=1e-6)
        again = part.lookup(ctx, torch.empty_like(got).to(DEV)).cpu()
        assert torch.equal(again, got)
        for r, n in batch:
            at[r] += n
        for r in end:
            h.cm.release(r)


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,dk,dv,ra,rg,n,parts", [(4, 12, 10, 5, 7, 40, 1), (2, 64, 32, 8, 16, 300, 1), (3, 18, 6, 1, 33, 9, 3), (16, 128, 128, 128, 64, 130, 1),
                                                   (5, 20, 36, 72, 24, 65, 1), (1, 7, 5, 3, 2, 1, 2)])
def test_low_rank_maps_alone(dt, H, dk, dv, ra, rg, n, parts):
    """Decays between nearly 0 and nearly 1 and the gate's sums, from one set of product sums or several parts; ranks and channel
    counts that are no multiples of any tile; the tensor-core form above 64 tokens."""
    g = torch.Generator().manual_seed(H + dk + n)
    off_a, off_g, off_b = 3, 5 + ra, 6 + ra + rg
    sums = torch.randn(parts, n, off_b + H + 2, generator=g) / parts ** 0.5
    a2, g2 = (torch.randn(H * dk, ra, generator=g) / ra ** 0.5).to(dt), (torch.randn(H * dv, rg, generator=g) / rg ** 0.5).to(dt)
    bias, a_log = 2.0 * torch.randn(H * dk, generator=g), torch.rand(H, generator=g) * 5.3 - 4.6
    decay = torch.empty(n, H * dk, device=DEV)
    gate, beta = torch.empty(n, H * dv, device=DEV), torch.empty(n, H, device=DEV)
    a2d, g2d = a2.to(DEV), g2.to(DEV)
    get_ops().channel_gates(sums.to(DEV), off_a, ra, off_g, rg, off_b, a2d.t().contiguous(), g2d.t().contiguous(), bias.to(DEV), a_log.to(DEV), decay,
                            gate, beta, n, decay_w=a2d, gate_w=g2d)
    s = sums.double().sum(0)
    w = {"a1": torch.eye(ra, dtype=torch.float64), "a2": a2.double(), "dt_bias": bias.double(), "A_log": a_log.double()}
    want = P.channel_decay(s[:, off_a:off_a + ra], w, "", H, dk).reshape(n, -1)
    np.testing.assert_allclose(decay.cpu().double().numpy(), want.numpy(), rtol=2e-4, atol=2e-5)   # both precisions: the numbers are float32
    np.testing.assert_allclose(beta.cpu().double().numpy(), P.sigmoid(s[:, off_b:off_b + H]).numpy(), rtol=1e-5)
    np.testing.assert_allclose(gate.cpu().double().numpy(), (s[:, off_g:off_g + rg] @ g2.double().T).numpy(), rtol=2e-4, atol=1e-4)


DELTA_CASES = [(ZUDATAR_A, 1), (ZUDATAR_A, 4), (ZUDATAR_B, 0), (ZUDATAR_B, 3), (ZUDATAR_C, 2),
               (one_layer(layer("channel_delta", delta(4, 4, 128, 128, 4)), width=96), 0), (one_layer(layer("channel_delta", delta(6, 3, 100, 36, 5))), 0),
               (one_layer(layer("channel_delta", delta(2, 2, 16, 130, 2))), 0)]


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("cfg,i", DELTA_CASES, ids=["a1", "a4", "b0", "b3", "c2", "128x128", "100x36", "16x130"])
def test_delta_rule_with_a_decay_a_channel_alone(dt, cfg, i):
    """Portions of 1, 2 and many tokens that hand the state and the convolutions' inputs on through the slot; one to five taps; heads
    that share queries and keys; key sizes that fill a part of a lane's numbers and several lanes."""
    cpu, dev, spec = layer_tensors(cfg, i, dt)
    part, h, cache = loaded("mixer", dt, spec.mixer, dev)
    m, state = cfg["layers"][i]["mixer"], {}
    x = torch.randn(140, cfg["width"], generator=torch.Generator().manual_seed(16)).to(dt)
    run_in_portions(part, h, cache, x, lambda xs: P.channel_delta(xs, cpu, f"l{i}.mix.", m, cfg["norm"]["eps"], state), dt)


def test_delta_rule_for_requests_side_by_side():
    """Portions of three requests in one step, short ones and long ones (runs of the convolution that cross a request's first
    token), each against itself alone."""
    dt = torch.float32
    cfg, i = ZUDATAR_B, 0
    cpu, dev, spec = layer_tensors(cfg, i, dt)
    part, h, cache = loaded("mixer", dt, spec.mixer, dev)
    m, g = cfg["layers"][i]["mixer"], torch.Generator().manual_seed(2)
    x = {r: torch.randn(120, cfg["width"], generator=g) for r in (1, 2, 3)}
    st, at = {r: {} for r in x}, {r: 0 for r in x}
    for batch in ([(1, 3), (2, 70), (3, 2)], [(3, 41), (1, 2), (2, 1)], [(2, 1), (3, 1), (1, 1)], [(1, 65), (2, 9), (3, 30)]):
        xs = torch.cat([x[r][at[r]:at[r] + n] for r, n in batch])
        got = whole(part.forward(xs.to(DEV), h.ctx([(r, n, []) for r, n in batch]), cache)).cpu()
        lo = 0
        for r, n in batch:
            want = P.channel_delta(x[r][at[r]:at[r] + n].double(), cpu, f"l{i}.mix.", m, 1e-6, st[r])
            close(got[lo:lo + n], want, dt, f"request {r} from {at[r]}")
            lo, at[r] = lo + n, at[r] + n


@pytest.mark.parametrize("dt", DTYPES)
def test_a_state_written_once_is_read_hundreds_of_tokens_later(dt):
    """Decays of nearly one (a very negative A_log and step) and a query that asks for one early token's key: what that token wrote is
    read 400 tokens later, after portions and single tokens; a state that is lost, reset or read from another slot on the way shows.
    Single taps, so that the early key and the late query are made of one token each; weak writes everywhere else."""
    cfg = one_layer(layer("channel_delta", delta(2, 2, 32, 48, 1)))
    cpu, dev, spec = layer_tensors(cfg, 0, dt)
    p = "l0.mix."
    b = torch.zeros_like(cpu[p + "b"])
    b[:, 0] = 8.0                                           # beta rests on the first number of the input alone
    for name, w in ((p + "A_log", torch.full((2,), -9.0)), (p + "b", b), (p + "q", cpu[p + "k"])):
        cpu[name], dev[name] = w.to(dt).double(), w.to(DEV, dev[name].dtype)
    part, h, cache = loaded("mixer", dt, spec.mixer, dev)
    m, T = cfg["layers"][0]["mixer"], 430
    x = torch.randn(T, cfg["width"], generator=torch.Generator().manual_seed(3))
    x[:, 0] = -1.0                                          # beta = sigmoid(-8)
    x[3, 0] = 1.0                                           # token 3 writes
    x[T - 2, 1:] = x[3, 1:]                                 # and token T - 2 asks along the same directions
    x = x.to(dt)
    want = P.channel_delta(x.double(), cpu, p, m, 1e-5, {})
    got, lo = [], 0
    for n in (2, 1, 1, 130, 1, 2, 200, 61, 1, 1, 30):
        got.append(whole(part.forward(x[lo:lo + n].to(DEV), h.ctx([(1, n, [])]), cache)).cpu())
        lo += n
    assert lo == T
    close(torch.cat(got), want, dt, "portions", tol32=2e-4)
    fresh = P.channel_delta(x[10:].double(), cpu, p, m, 1e-5, {})  # the same tokens without what token 3 wrote
    assert float((fresh[T - 12] - want[T - 2]).norm()) > 0.3 * float(want[T - 2].norm()), "the case is meant to depend on token 3"


def _attention(heads, kv_heads, dim, window, rot):
    return one_layer(layer("attention", att(heads, kv_heads, dim, dim ** -0.5, window, rot)))


ATTENTION_CASES = [(ZUDATAR_A, 2), (ZUDATAR_B, 1), (ZUDATAR_B, 5), (ZUDATAR_C, 0), (ZUDATAR_C, 4), (_attention(8, 1, 128, 300, (64, 5e5)), 0),
                   (_attention(2, 2, 32, 7, (32, 100.0)), 0), (_attention(6, 2, 96, 30, (24, 1e4)), 0), (_attention(2, 1, 300, 40, (2, 9.0)), 0)]


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("cfg,i", ATTENTION_CASES, ids=["a2", "b1", "b5", "c0", "c4", "128", "32", "96", "300"])
@pytest.mark.parametrize("sharp", [False, True])
def test_attention_alone(dt, cfg, i, sharp):
    """Over a prompt portion, then over single tokens and further portions that read the first one's cache rows: biases, pairs of
    neighbours over a part of a head, all of it and none, root mean squares behind the rotation, values that are the keys before
    both, a gate a head; windows shorter than a portion, of one page; head sizes of every attention kernel."""
    if sharp:
        cfg = sharpened(cfg)
    cpu, dev, spec = layer_tensors(cfg, i, dt)
    part, h, cache = loaded("mixer", dt, spec.mixer, dev)
    m, state = cfg["layers"][i]["mixer"], {}
    x = torch.randn(140, cfg["width"], generator=torch.Generator().manual_seed(6)).to(dt)
    run_in_portions(part, h, cache, x, lambda xs: P.attention(xs, cpu, f"l{i}.mix.", m, cfg["norm"]["eps"], state), dt)


def _latent(heads, dim, vdim, kv_rank, q_rank, window):
    return one_layer(layer("latent_attention", lat(heads, dim, vdim, kv_rank, q_rank, dim ** -0.5, window)))


LATENT_CASES = [(ZUDATAR_A, 0), (ZUDATAR_B, 2), (ZUDATAR_C, 1), (_latent(16, 64, 64, 128, 96, 50), 0), (_latent(3, 48, 24, 192, 40, 9), 0),
                (_latent(40, 16, 16, 64, 24, 33), 0), (_latent(2, 32, 32, 512, 16, 100), 0), (_latent(5, 20, 12, 30, 11, 64), 0)]


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("cfg,i", LATENT_CASES, ids=["a0", "b2", "c1", "128", "192", "40heads", "512", "30"])
@pytest.mark.parametrize("sharp", [False, True])
def test_latent_attention_alone(dt, cfg, i, sharp):
    """Sinks of both signs, windows, a gate a head, latents of the tensor-core kernel's sizes and others, more heads than a tile."""
    cpu, dev, spec = layer_tensors(cfg, i, dt, sharp)
    part, h, cache = loaded("mixer", dt, spec.mixer, dev)
    m, state = cfg["layers"][i]["mixer"], {}
    x = torch.randn(140, cfg["width"], generator=torch.Generator().manual_seed(7)).to(dt)
    run_in_portions(part, h, cache, x, lambda xs: P.latent_attention(xs, cpu, f"l{i}.mix.", m, cfg["norm"]["eps"], state), dt)


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("sink", [-40.0, 0.0, 12.0])
def test_sink_alone(dt, sink):
    """A sink that nothing notices, one that counts as a key with a score of zero, one that takes nearly all the weight; a first
    token (whose only other term is its own) in a prompt and decoded."""
    cfg = one_layer(layer("latent_attention", lat(4, 32, 24, 64, 20, 0.2, 6)))
    cpu, dev, spec = layer_tensors(cfg, 0, dt)
    cpu["l0.mix.sink"] = torch.full((4,), sink, dtype=torch.float64)
    dev["l0.mix.sink"] = torch.full((4,), sink, device=DEV)
    part, h, cache = loaded("mixer", dt, spec.mixer, dev)
    state = {}
    x = torch.randn(30, cfg["width"], generator=torch.Generator().manual_seed(9)).to(dt)
    run_in_portions(part, h, cache, x, lambda xs: P.latent_attention(xs, cpu, "l0.mix.", cfg["layers"][0]["mixer"], 1e-5, state), dt,
                    ((0, 1), (1, 2), (2, 20), (20, 21), (21, 30)))


def _probe(cpu, dev, p, kind, m, dt):
    """Weights with which a token whose input has its first number set looks for the tokens whose input has the second one set: one
    direction of the query meets one direction of the key, with a score that stands far out. Attention: the biases hold the norms
    behind the rotation apart from zero, and the probing numbers lie outside the rotated part."""
    H = m["heads"]
    if kind == "attention":
        G, dk = m["kv_heads"], m["dim"]
        q, k, qb, kb = (torch.zeros_like(cpu[p + s]) for s in ("q", "k", "q.b", "k.b"))
        q[dk - 1::dk, 0] = 8.0                               # asks along the head's last number
        qb[dk - 2::dk] = 1.0                                 # and otherwise along one where every key is zero
        k[dk - 1::dk, 1] = 8.0
        kb[dk - 3::dk] = 1.0
        k[torch.arange(G * dk) % dk < dk - 3] = cpu[p + "k"][torch.arange(G * dk) % dk < dk - 3] * 0.05   # what the values carry
        new = {"q": q, "k": k, "q.b": qb, "k.b": kb}
    else:
        dk, R, Rq = m["dim"], m["kv_rank"], m["q_rank"]
        dq, uq, uk = (torch.zeros_like(cpu[p + s]) for s in ("dq", "uq", "uk"))
        dq[0, 0], dq[1, 2] = 8.0, 1.0                        # the query latent: what is asked for, and something that is always there
        uq[0::dk, 0] = 1.0
        uk[0::dk, 0] = 60.0 / (m["scale"] * R ** 0.5 * Rq ** 0.5)
        new = {"dq": dq, "dq.norm": torch.ones(Rq), "uq": uq, "uk": uk, "sink": torch.zeros(H)}
        if p + "dkv" in cpu:
            dkv = cpu[p + "dkv"] * 0.1
            dkv[:, :3] = 0
            dkv[0], dkv[0, 1] = 0.0, 8.0                     # the latent's first number: the mark
            new.update({"dkv": dkv, "dkv.norm": torch.ones(R)})
    for s, w in new.items():
        cpu[p + s], dev[p + s] = w.to(dt).double(), w.to(DEV, dev[p + s].dtype)


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("window,page", [(13, 4), (16, 16), (40, 16), (1, 4), (300, 16)])
@pytest.mark.parametrize("decoded", [False, True])
@pytest.mark.parametrize("kind", ["attention", "latent", "borrowed"])
def test_a_marked_key_just_inside_and_just_outside_the_window(dt, window, page, decoded, kind):
    """Hundreds of tokens of which one is marked; later tokens ask for it with a score that stands far out. The one that is
    `window - 1` behind it sees it, the next one does not; the same when the asking tokens are decoded one by one, when the marked key
    lies on a page's last or first row, and when the asking layer reads another layer's latents (whose own window is a different
    one). What the plain implementation computes with a window that is one token off must lie far from it."""
    if kind == "attention":
        layers = [layer("attention", att(4, 2, 16, 16 ** -0.5 * 4, window, (8, 100.0)))]
    else:
        first = layer("latent_attention", lat(4, 16, 24, 64, 12, 0.25, 5 if kind == "borrowed" else window))
        layers = [first] + ([layer("latent_attention", lat(4, 16, 24, 64, 12, 0.25, window, kv_from=0))] if kind == "borrowed" else [])
    cfg = one_layer(layers[-1], before=layers[:-1])
    plain_kind = "attention" if kind == "attention" else "latent"
    mixers = [l["mixer"] for l in layers]
    sides, T = [], 420
    for i, m in enumerate(mixers):
        cpu, dev, spec = layer_tensors(cfg, i, dt)
        _probe(cpu, dev, f"l{i}.mix.", plain_kind, m, dt)
        sides.append((cpu, dev, spec))
    owner, h, cache = loaded("mixer", dt, sides[0][2].mixer, sides[0][1], page=page, pages=T // page + 4)
    assert owner.cache_needs()[0].window == (max(5, window) if kind == "borrowed" else window)
    asker = owner
    if kind == "borrowed":
        asker = build_part("mixer", sides[1][2].mixer, h.env)
        asker.load(sides[1][1])
        assert not asker.cache_needs()
    read = LayerCache(group=0, k=cache.k, v=cache.v, writes=False, window=cache.window)

    def plain(x, m_last):
        if kind == "attention":
            return P.attention(x, sides[0][0], "l0.mix.", m_last, 1e-5, {})
        st = {}
        y = P.latent_attention(x, sides[0][0], "l0.mix.", mixers[0] if kind == "borrowed" else m_last, 1e-5, st)
        return P.latent_attention(x, sides[1][0], "l1.mix.", m_last, 1e-5, {}, st) if kind == "borrowed" else y

    for marked in (page * 5 - 1, page * 5, 77):
        x = torch.randn(T, cfg["width"], generator=torch.Generator().manual_seed(marked))
        x[:, :2] = 0
        x[:, 2] = 1.0
        x[marked, 1] = 1.0                       # the key that is looked for
        x[marked, 3:] *= 3.0                     # and what it carries
        for a in (marked + window - 1, marked + window, marked + 150):
            if a < T and a != marked:
                x[a, 0] = 1.0
        x = x.to(dt)
        want = plain(x.double(), mixers[-1])
        cut = marked + 1 if decoded else T
        steps = [(0, cut)] + [(t, t + 1) for t in range(cut, min(T, marked + window + 2))]
        got = []
        for lo, hi in steps:
            ctx = h.ctx([(marked + 1, hi - lo, [])])
            y = owner.forward(x[lo:hi].to(DEV), ctx, cache)
            if kind == "borrowed":
                y = asker.forward(x[lo:hi].to(DEV), ctx, read)
            got.append(whole(y).cpu())
        got = torch.cat(got)
        close(got, want[:got.shape[0]], dt, f"marked key at {marked}")
        h.cm.release(marked + 1)
        for off, row in ((-1, marked + window - 1), (1, marked + window)):   # windows one token shorter and longer differ where it matters
            if window + off >= 1 and row < T and row != marked:
                other = plain(x[:row + 1].double(), dict(mixers[-1], mask={"size": window + off}))
                assert float((other[row] - want[row]).norm()) > 0.3 * float(want[row].norm()), (off, row)


@pytest.mark.parametrize("dt", DTYPES)
def test_a_borrower_keeps_its_own_maps_queries_and_sink(dt):
    """Owner and reader in portions: the reader has heads, sizes, window, sink and gate of its own; it writes nothing."""
    for cfg, (i, j) in ((ZUDATAR_A, (0, 3)), (ZUDATAR_B, (2, 4)), (ZUDATAR_C, (1, 3)), (ZUDATAR_C, (1, 5))):
        sharp = dt == torch.float32  # (in bfloat16 the rounding of queries moves sharp scores by more than the comparison allows)
        ci, di, si = layer_tensors(cfg, i, dt, sharp)
        cj, dj, sj = layer_tensors(cfg, j, dt, sharp)
        owner, h, cache = loaded("mixer", dt, si.mixer, di)
        reader = build_part("mixer", sj.mixer, h.env)
        reader.load(dj)
        read = LayerCache(group=0, k=cache.k, v=None, writes=False, window=cache.window)
        mi, mj, eps = cfg["layers"][i]["mixer"], cfg["layers"][j]["mixer"], cfg["norm"]["eps"]
        g = torch.Generator().manual_seed(21)
        x, y = torch.randn(140, cfg["width"], generator=g).to(dt), torch.randn(140, cfg["width"], generator=g).to(dt)
        a, b = {}, {}
        for lo, hi in PORTIONS:
            ctx = h.ctx([(1, hi - lo, [])])
            owner.forward(x[lo:hi].to(DEV), ctx, cache)
            P.latent_attention(x[lo:hi].double(), ci, f"l{i}.mix.", mi, eps, a)
            before = cache.k.clone()
            got = whole(reader.forward(y[lo:hi].to(DEV), ctx, read)).cpu()
            assert torch.equal(before, cache.k)
            close(got, P.latent_attention(y[lo:hi].double(), cj, f"l{j}.mix.", mj, eps, b, a), dt, f"layers {i} and {j}, positions {lo}..{hi}")
        with pytest.raises(RuntimeError):
            reader.forward(y[:1].to(DEV), ctx, LayerCache())


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("cfg,i", [(ZUDATAR_A, 0), (ZUDATAR_A, 1), (ZUDATAR_A, 2), (ZUDATAR_B, 0), (ZUDATAR_B, 1), (ZUDATAR_B, 2), (ZUDATAR_C, 4)],
                         ids=["a0", "a1", "a2", "b0", "b1", "b2", "c4"])
def test_block_alone(dt, cfg, i):
    """A whole layer on a float32 stream: a norm before and one after each sub-layer; a layer without a feed-forward."""
    from llmengine.parts.base import Residual
    cpu, dev, spec = layer_tensors(cfg, i, dt)
    block, h, cache = loaded("block", dt, spec, dev)
    eps, l, p = cfg["norm"]["eps"], cfg["layers"][i], f"l{i}."
    x = torch.randn(60, cfg["width"], generator=torch.Generator().manual_seed(46)) + 0.5
    state, lo = {}, 0
    mix = {"channel_delta": P.channel_delta, "attention": P.attention, "latent_attention": P.latent_attention}[l["type"]]
    for n in (17, 1, 2, 40):
        want = x[lo:lo + n].double()
        want = want + P.rms(mix(P.rms(want, eps) * cpu[p + "norm1"], cpu, p + "mix.", l["mixer"], eps, state), eps) * cpu[p + "norm1b"]
        if l["mlp"]:
            want = want + P.rms(P.dense_ff(P.rms(want, eps) * cpu[p + "norm2"], cpu, p + "mlp."), eps) * cpu[p + "norm2b"]
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


@pytest.fixture(scope="module", params=[(n, dt, sharp) for n in ("za", "zb", "zc") for dt in DTYPES for sharp in (False, True)
                                        if not (sharp and n == "zc")],
                ids=lambda p: f"{p[0]}-{NAMES[p[1]]}{'-sharp' if p[2] else ''}")
def model(request, tmp_path_factory):
    name, dt, sharp = request.param
    cfg, page = ZUDATAR[name]
    d = write_model(str(tmp_path_factory.mktemp("zudatar")), cfg, dt, sharp=sharp)
    pc, pw = P.read_model(d)
    lens = [5, 64, 33, 130, 97] if name != "zb" else [3, 47, 64, 200, 129]
    reqs = {f"r{i}": random_ids(n, cfg["vocab"], 50 + i) for i, n in enumerate(lens)}
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


def test_keys_at_page_borders_window_edges_and_first_tokens(model):
    """A request that grows one token a step from its first token across page borders and past every window's length, beside a
    second one that starts later (so that its pages lie between the first one's, and its state in another slot)."""
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
        close(lg[lo:lo + n], alone, dt, f"{k}: batch against alone", tol32=2e-5, tol16=3e-2)
        lo += n


def test_a_slot_that_is_used_again_starts_at_zero(model):
    """Requests one after the other in an engine with a single live request at a time: each gets the one before's slot and pages,
    and must not see its state, its previous token or its keys."""
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
    for p in range(10, 100):  # the chosen token is the plain logits' best, or ties with it within rounding
        assert logits[p, out[p + 1]] >= logits[p].max() - slack * max(1.0, np.abs(logits[p]).max()), p


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("dim,rank,window", [(64, 64, 136), (64, 128, 1400), (128, 512, 700), (48, 48, 136)])
def test_single_tokens_behind_long_contexts(dt, dim, rank, window, tmp_path):
    """Three requests of unequal length (up to 1,500 tokens) whose last tokens come one a step, side by side: single tokens whose
    key range is cut into pieces that run side by side and are merged, windows that end inside a piece and windows longer than a
    request; a reader of the latents with a window of its own and a delta layer behind them."""
    layers = [layer("attention", att(4, 2, dim, 6.0 / dim ** 0.5, window, (dim // 2, 1e4)), 64),
              layer("latent_attention", lat(4, 32, 16, rank, 24, 0.2, window), 48),
              layer("channel_delta", delta(2, 1, 32, 48, 4)),
              layer("latent_attention", lat(3, 24, 32, rank, 20, 0.2, 90, kv_from=1))]
    cfg = config(120, 64, 1e-5, 3.0, (199, 7, 11), 0.7, layers, 2048)
    d = write_model(str(tmp_path / "m"), cfg, dt, sharp=True)
    pc, pw = P.read_model(d)
    reqs = {"a": random_ids(1500, 120, 1), "b": random_ids(700, 120, 2), "c": random_ids(200, 120, 3)}
    tail = 24
    eng = llmengine.Engine(d, NAMES[dt], block_size=16)
    eng.configure_cache(num_blocks=(1536 + 704 + 256) // 16, block_size=16, num_slots=4)
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
@pytest.mark.parametrize("name", ["za", "zb"])
def test_replay_through_the_command(dtype, name, tmp_path):
    """bin/trace_run as a user runs it."""
    cfg, page = ZUDATAR[name]
    dt = torch.float32 if dtype == "float32" else torch.bfloat16
    d = write_model(str(tmp_path / "m"), cfg, dt)
    pc, pw = P.read_model(d)
    reqs = {f"q{i}": random_ids(n, cfg["vocab"], 80 + i) for i, n in enumerate([2, 70, 35, 150])}
    t = trace_mixed(reqs, 256 + 64, seed=3, sizes=MIXED_SIZES_LONG)
    rows = run_trace(d, dtype, t, str(tmp_path / "out"), 256 + 64, page, cfg["vocab"])
    for k, ids in reqs.items():
        rows_close(np.stack([rows[(k, p)] for p in range(len(ids))]), P.forward(pc, pw, ids).numpy(), dt, k,
                   rounded_forward(pc, pw, ids) if dtype == "bfloat16" else None)


def test_generation_from_the_command_line(tmp_path):
    from test_cli import run_cli
    d = write_model(str(tmp_path / "model"), ZUDATAR_C, torch.float32)
    r = run_cli("--model", d, "--prompt-ids", "5,17,3,90", "--max-new", "6", "--block-size", "8", "--num-blocks", "32")
    assert r.returncode == 0, r.stderr
    line = [json.loads(l) for l in r.stdout.splitlines() if l.startswith("{")][0]
    pc, pw = P.read_model(d)
    assert line["token_ids"] == P.greedy(pc, pw, [5, 17, 3, 90], 6) and line["finish_reason"] == "length"
