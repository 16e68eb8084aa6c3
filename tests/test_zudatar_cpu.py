"""Zudatar without a GPU: configuration and its errors, the description in parts (tensor names, which run reads whose latents, how
many latents a cache keeps for its readers, sizes and ranks that tensor shapes give), the random-weights mode, the plain
implementation against itself and against cases made by hand, and the engine's host side on the test double of the kernels (the
embedding's own state among it)."""
import copy
import json
import math

import numpy as np
import pytest
import torch

import llmengine
import plain_zudatar as P
from llmengine.config import ConfigError
from llmengine.config.registry import config_from_dir, get_architecture
from llmengine.config.zudatar import ZudatarConfig, sizes_from_tensors
from llmengine.models.zudatar import describe_zudatar, kept_window
from llmengine.weights.random_init import model_tensor_needs
from cpu_ops import CpuOps
from tiny import random_ids
from tiny_zudatar import RANKS, ZUDATAR, ZUDATAR_A, ZUDATAR_B, ZUDATAR_C, make_tensors, write_model


def with_ranks(name):
    """config.json with the ranks written out, as the random-weights mode writes it."""
    c = copy.deepcopy(ZUDATAR[name][0])
    for i, (a, g) in RANKS[name].items():
        c["layers"][i]["mixer"].update(decay_rank=a, gate_rank=g)
    return c


@pytest.mark.parametrize("name", sorted(ZUDATAR))
def test_configuration_round_trip_and_tensor_names(name):
    cfg = with_ranks(name)
    c = ZudatarConfig.from_dict(cfg)
    assert ZudatarConfig.from_dict(c.to_dict()) == c
    assert get_architecture("Zudatar").parse_config(cfg, None) == c
    spec = describe_zudatar(c)
    needs = model_tensor_needs(spec)
    made = make_tensors(ZUDATAR[name][0], 1, torch.float32)
    assert set(needs) == set(made)
    for k, n in needs.items():
        assert tuple(made[k].shape) == tuple(n.shape), k
    assert [b.kind for b in spec.layers] == ["sandwich"] * len(cfg["layers"])
    assert [r.layer for r in spec.order] == list(range(len(cfg["layers"])))
    assert [r.cache_from for r in spec.order] == [l["mixer"].get("kv_from") for l in cfg["layers"]]


def test_description_reads_every_option():
    spec = describe_zudatar(ZudatarConfig.from_dict(with_ranks("za")))
    l0, d1, a2, l3, d4 = (b.mixer for b in spec.layers)
    e = spec.embedding
    assert (e.kind, e.weight, e.scale, e.pair_weight, e.pair_buckets, e.pair_mul_prev, e.pair_mul_cur) == ("lookup_pairs", "embed", 3.7, "bigram", 53, 17, 5)
    assert spec.head.weight == "embed" and spec.final_norm.gain == 1.9 and spec.layers[0].norm1.gain == 1.0
    assert (l0.kind, l0.heads, l0.dim, l0.rot_dim, l0.vdim, l0.kv_rank, l0.q_rank, l0.scale, l0.window) == ("latent_attention", 3, 10, 0, 14, 18, 22, 0.4, 7)
    assert l0.own_kv and l0.sink == "l0.mix.sink" and l0.gate_per_head and l0.cache_window == 21
    assert not l3.own_kv and l3.dkv_weight is None and l3.window == 21 and l3.cache_window is None
    assert (d1.kind, d1.heads, d1.kv_heads, d1.dim, d1.vdim, d1.taps, d1.decay_rank, d1.gate_rank) == ("channel_delta", 4, 2, 12, 10, 3, 5, 7)
    assert d4.taps == 1 and d1.unit_eps == 1e-6 and d1.eps == 1e-5
    assert (a2.num_heads, a2.num_kv_heads, a2.head_dim, a2.value_dim, a2.scale, a2.window) == (6, 2, 18, 18, 0.21, 13)
    assert a2.keys_as_values and a2.unit_rms and a2.rot_pairs == "neighbours" and a2.gate_per_head and a2.v_weight is None
    assert (a2.q_bias, a2.k_bias, a2.position.dims, a2.position.base) == ("l2.mix.q.b", "l2.mix.k.b", 8, 777.0)
    assert spec.layers[2].feed_forward is None and spec.layers[2].norm2 is None and "l2.norm2" in spec.ignore
    assert spec.layers[0].feed_forward.activation == "silu" and spec.layers[0].residual_mult == 1.0


def test_a_cache_keeps_what_its_widest_reader_asks_for():
    a, b, c = (ZudatarConfig.from_dict(ZUDATAR[n][0]) for n in ("za", "zb", "zc"))
    assert kept_window(a, 0) == 21 and kept_window(b, 2) == 40 and kept_window(c, 1) == 30
    from llmengine.engine.model import Model
    from llmengine.parts.base import BuildEnv
    m = Model(describe_zudatar(b), BuildEnv(torch.device("cpu"), torch.float32, CpuOps(), 16))
    assert sorted(m.windows) == [24, 40, 48] and m.run_group[4] is None and m.run_needs[4] == ()
    assert [n.name for n in m.embedding_needs] == ["embedding.previous"]


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][2]["mixer"].update(heads=5), "multiple of kv_heads"),
    (lambda c: c["layers"][1]["mixer"].update(heads=5), "multiple of kv_heads"),
    (lambda c: c["layers"][2]["mixer"].update(vdim=12), "the values are the keys"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=7), "even"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=20), "at most dim"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=1), "no earlier latent_attention layer"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=3), "no earlier latent_attention layer"),
    (lambda c: c["layers"][3]["mixer"].update(kv_rank=16), "kv_rank"),
    (lambda c: c["layers"][0].update(type="conv"), "unknown layer type"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "unknown kind"),
    (lambda c: c["layers"][0]["mlp"].update(ff=0), "ff must be positive"),
    (lambda c: c["embedding"]["bigram"].update(buckets=0), "buckets"),
    (lambda c: c["embedding"]["bigram"].pop("mul_cur"), "mul_cur"),
    (lambda c: c.pop("width"), "width"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
])
def test_configuration_errors(change, message):
    cfg = copy.deepcopy(ZUDATAR_A)
    change(cfg)
    with pytest.raises(ConfigError) as e:
        ZudatarConfig.from_dict(cfg)
    assert message in str(e.value)


def test_a_layer_cannot_read_a_readers_latents():
    cfg = copy.deepcopy(ZUDATAR_C)
    cfg["layers"][5]["mixer"]["kv_from"] = 3
    with pytest.raises(ConfigError) as e:
        ZudatarConfig.from_dict(cfg)
    assert "no latents of its own" in str(e.value)


def test_sizes_that_only_tensor_shapes_give(tmp_path):
    """The ranks of the low-rank maps, which no configuration names, and every other size left out of a file."""
    write_model(str(tmp_path / "m"), ZUDATAR_A, torch.float32)
    arch, parsed = config_from_dir(str(tmp_path / "m"))
    assert parsed == ZudatarConfig.from_dict(with_ranks("za"))
    cfg = copy.deepcopy(ZUDATAR_A)
    del cfg["vocab"], cfg["width"], cfg["embedding"]["bigram"]["buckets"]
    for l in cfg["layers"]:
        for key in ("heads", "kv_heads", "dim", "vdim", "conv", "kv_rank", "q_rank"):
            l["mixer"].pop(key, None)
        if l["mlp"]:
            del l["mlp"]["ff"]
    with open(tmp_path / "m" / "config.json", "w") as f:
        json.dump(cfg, f)
    assert config_from_dir(str(tmp_path / "m"))[1] == parsed
    assert sizes_from_tensors(ZUDATAR_B, lambda name: (1, 1))["layers"][1] == ZUDATAR_B["layers"][1]   # what the file says stays


def test_random_weights_mode(tmp_path):
    d = llmengine.write_random_model(str(tmp_path / "m"), ZUDATAR_B, seed=3, dtype=torch.bfloat16)
    arch, parsed = config_from_dir(d)
    assert arch.name == "Zudatar" and len(parsed.layers) == 6 and parsed.layers[0].mixer.decay_rank == 16
    names = set(P.read_safetensors(str(tmp_path / "m" / "model.safetensors")))
    assert names >= {"embed", "bigram", "final.norm", "l0.mix.a1", "l0.mix.g2", "l1.mix.k.b", "l2.mix.sink", "l4.mix.uk"}
    assert not names & {"l1.mix.v", "l4.mix.dkv", "l4.mix.dkv.norm", "l3.norm2", "embed.norm"}


# ---------------------------------------------------------------------------------------------- the plain rules by hand
def test_plain_pair_embedding_by_hand():
    w = {"embed": torch.arange(6, dtype=torch.float64)[:, None], "bigram": 100.0 * torch.arange(8, dtype=torch.float64)[:, None]}
    e = {"scale": 2.0, "bigram": {"buckets": 7, "mul_prev": 3, "mul_cur": 5}}
    st = {}
    x = P.embedding([4, 1], w, e, st)
    assert x[0, 0] == 8 + 700 and x[1, 0] == 2 + 100 * ((4 * 3 + 1 * 5) % 7)   # the first token takes the last row
    x = P.embedding([5], w, e, st)
    assert x[0, 0] == 10 + 100 * ((1 * 3 + 5 * 5) % 7)                          # the previous token is part of the state


def test_plain_rotation_of_neighbours_by_hand():
    x = torch.tensor([[1.0, 2.0, 3.0, 4.0, 5.0]], dtype=torch.float64)
    y = P.rotate_neighbours(x, 3, {"dims": 4, "base": 100.0})
    for i in range(2):
        a = 3 * 100.0 ** (-2.0 * i / 4)
        u, v = float(x[0, 2 * i]), float(x[0, 2 * i + 1])
        assert math.isclose(float(y[0, 2 * i]), u * math.cos(a) - v * math.sin(a))
        assert math.isclose(float(y[0, 2 * i + 1]), v * math.cos(a) + u * math.sin(a))
    assert y[0, 4] == 5.0


def test_plain_sink_and_window_by_hand():
    p = P.softmax_with_sink(torch.tensor([0.0, 1.0], dtype=torch.float64), torch.tensor(2.0, dtype=torch.float64))
    z = 1 + math.e + math.e ** 2
    assert math.isclose(float(p[0]), 1 / z) and math.isclose(float(p[1]), math.e / z)
    assert [P.first_visible(i, 3) for i in range(5)] == [0, 0, 0, 1, 2]


def test_plain_delta_step_by_hand():
    """One head of two channels: the state decays a channel at a time first, the write sees the decayed state, the read sees the write."""
    S = torch.tensor([[[2.0], [4.0]]], dtype=torch.float64)
    k, q = torch.tensor([[1.0, 0.0]], dtype=torch.float64), torch.tensor([[1.0, 10.0]], dtype=torch.float64)
    S2, o = P.delta_step(S, q, k, torch.tensor([[5.0]], dtype=torch.float64), torch.tensor([[0.5, 0.25]], dtype=torch.float64),
                         torch.tensor([0.5], dtype=torch.float64))
    assert S2[0, :, 0].tolist() == [1.0 + 0.5 * (5.0 - 1.0), 1.0] and o[0, 0] == 3.0 + 10.0


def test_plain_values_are_the_keys_before_norm_and_rotation():
    w = {"q": torch.zeros(2, 2, dtype=torch.float64), "q.b": torch.tensor([1.0, 0.0], dtype=torch.float64), "k": 3.0 * torch.eye(2, dtype=torch.float64),
         "k.b": torch.tensor([0.0, 1.0], dtype=torch.float64), "g": torch.zeros(1, 2, dtype=torch.float64), "o": torch.eye(2, dtype=torch.float64)}
    m = {"heads": 1, "kv_heads": 1, "dim": 2, "scale": 0.0, "mask": {"size": 9}, "rot": {"dims": 2, "base": 10.0}}
    h = torch.tensor([[1.0, 0.0], [0.0, 1.0]], dtype=torch.float64)
    y = P.attention(h, w, "", m, 1e-9, {})
    assert torch.allclose(y[0], 0.5 * torch.tensor([3.0, 1.0], dtype=torch.float64))   # one gate a head: sigmoid(0)
    assert torch.allclose(y[1], 0.5 * torch.tensor([1.5, 2.5], dtype=torch.float64))   # scale 0: the mean of (3, 1) and (0, 4)


@pytest.mark.parametrize("name", sorted(ZUDATAR))
def test_plain_whole_against_portions_and_single_tokens(name):
    cfg = ZUDATAR[name][0]
    w = {k: v.double() for k, v in make_tensors(cfg, 2, torch.float32).items()}
    ids = random_ids(45, cfg["vocab"], 7)
    want = P.forward(cfg, w, ids)
    m = P.Plain(cfg, w)
    got = torch.cat([m.run(ids[a:b]) for a, b in ((0, 1), (1, 3), (3, 20), (20, 21), (21, 45))])
    assert float((got - want).abs().max()) < 1e-9


# ---------------------------------------------------------------------------------------------- the engine's host side
@pytest.fixture(scope="module", params=["za", "zc"])
def cpu_engine(request, tmp_path_factory):
    """The engine on the test double of the kernels: batch building, block tables (a window's pages given back while a reader with a
    wider window still needs them), state slots of layers and of the embedding, the wiring of the parts."""
    cfg, page = ZUDATAR[request.param]
    d = write_model(str(tmp_path_factory.mktemp("zudatar_" + request.param)), cfg, torch.float32, sharp=True)
    eng = llmengine.Engine(d, "fp32", device="cpu", ops=CpuOps(), block_size=page, num_blocks=40)
    eng.configure_cache(num_blocks=40, block_size=page, num_slots=3)
    return eng, P.read_model(d), cfg


def test_engine_on_the_test_double_matches_plain(cpu_engine):
    eng, (pc, pw), cfg = cpu_engine
    a, b = random_ids(37, cfg["vocab"], 1), random_ids(11, cfg["vocab"], 2)
    want = {k: P.forward(pc, pw, ids).numpy() for k, ids in (("a", a), ("b", b))}
    got = eng.run_step([(1, a, list(range(len(a))))], end=[1]).numpy()
    assert np.abs(got - want["a"]).max() < 2e-4
    rows = {}
    steps = [([(2, a[:9], [8]), (3, b[:10], [9])], []), ([(2, a[9:11], [0, 1]), (3, b[10:], [0])], [3]),
             ([(2, a[11:36], [24]), (4, b[:3], [2])], []), ([(2, a[36:], [0]), (4, b[3:], [7])], [2, 4])]
    at = {2: 0, 3: 0, 4: 0}
    for batch, end in steps:
        lg = eng.run_step(batch, end=end).numpy().copy()
        i = 0
        for rid, toks, w in batch:
            for k in w:
                rows[(rid, at[rid] + k)] = lg[i]
                i += 1
            at[rid] += len(toks)
    for (rid, pos), row in rows.items():
        ref = want["a"] if rid == 2 else want["b"]
        assert np.abs(row - ref[pos]).max() < 2e-4, (rid, pos)
    assert eng.cm.num_requests == 0


def test_stream_after_every_layer_on_the_test_double(cpu_engine):
    eng, (pc, pw), cfg = cpu_engine
    ids = random_ids(23, cfg["vocab"], 4)
    want, got = [], []
    P.forward(pc, pw, ids, after_layers=want)
    model = eng._ensure_model()
    model.after_run = lambda r, h: got.append((r, h.clone()))
    try:
        eng.run_step([(8, ids, [len(ids) - 1])], end=[8])
    finally:
        model.after_run = None
    assert [r for r, _ in got] == list(range(len(cfg["layers"]))) and len(want) == len(got)
    for (r, a), b in zip(got, want):
        assert float((a.double() - b).abs().max()) < 2e-4 * max(1.0, float(b.abs().max())), r


def test_generation_through_the_scheduler_matches_plain(cpu_engine):
    eng, (pc, pw), cfg = cpu_engine
    prompt = random_ids(9, cfg["vocab"], 3)
    out, reason = eng.generate(prompt, 7)
    assert reason == "length" and out == P.greedy(pc, pw, prompt, 7)


def test_command_line_random_weights_mode(tmp_path):
    from test_cli import run_cli
    cfg = tmp_path / "c.json"
    cfg.write_text(json.dumps(ZUDATAR_B))
    out = tmp_path / "model"
    r = run_cli("--random-weights", str(out), "--config", str(cfg), "--seed", "4", "--dtype", "bf16")
    assert r.returncode == 0, r.stderr
    arch, parsed = config_from_dir(str(out))
    assert arch.name == "Zudatar" and len(parsed.layers) == 6
