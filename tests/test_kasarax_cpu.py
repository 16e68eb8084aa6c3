"""Kasarax without a GPU: configuration and its errors, the description in parts (tensor names, options, sizes that tensor shapes
give), the random-weights mode, the plain implementation against itself and against cases made by hand, and the engine's host side on
the test double of the kernels."""
import copy
import json
import math

import numpy as np
import pytest
import torch

import llmengine
import plain_kasarax as P
from llmengine.config import ConfigError
from llmengine.config.kasarax import KasaraxConfig, sizes_from_tensors
from llmengine.config.registry import config_from_dir, get_architecture
from llmengine.models.kasarax import describe_kasarax
from llmengine.parts.gated_attention import query_temperatures
from llmengine.parts.spec import QueryTemperatureSpec
from llmengine.weights.random_init import model_tensor_needs
from cpu_ops import CpuOps
from tiny import random_ids
from tiny_kasarax import KASARAX, KASARAX_A, KASARAX_B, KASARAX_C, make_tensors, write_model


@pytest.mark.parametrize("name", sorted(KASARAX))
def test_configuration_round_trip_and_tensor_names(name):
    cfg = KASARAX[name][0]
    c = KasaraxConfig.from_dict(cfg)
    assert KasaraxConfig.from_dict(c.to_dict()) == c
    assert get_architecture("Kasarax").parse_config(cfg, None) == c
    spec = describe_kasarax(c)
    needs = model_tensor_needs(spec)
    made = make_tensors(cfg, 1, torch.float32)
    assert set(needs) == set(made)
    for k, n in needs.items():
        assert tuple(made[k].shape) == tuple(n.shape), k
    assert [b.kind for b in spec.layers] == ["parallel"] * len(cfg["layers"])
    assert [(r.layer, r.cache_from) for r in spec.order] == [(i, None) for i in range(len(cfg["layers"]))]


def test_description_reads_every_option():
    spec = describe_kasarax(KasaraxConfig.from_dict(KASARAX_A))
    a0, p1, p2, a3 = (b.mixer for b in spec.layers)
    assert spec.embedding.kind == "lookup" and spec.head.weight == "embed" and spec.final_norm.gain == 1.9
    assert all(b.norm2 is None and b.norm1.kind == "rmsnorm_unit_offset" and b.norm1.gain == 1.0 for b in spec.layers)
    assert (a0.num_heads, a0.num_kv_heads, a0.head_dim, a0.value_dim, a0.scale, a0.window) == (6, 2, 18, 10, 0.25, 0)
    assert (a0.q_bias, a0.k_bias, a0.v_bias, a0.o_bias) == tuple(f"l0.mix.{s}.b" for s in "qkvo")
    assert a0.sink is None and a0.sink_score == 0.0 and a0.gate_weight == "l0.mix.g" and a0.gate_per_head and a0.position.dims == 0
    assert (a0.q_temperature.coef, a0.q_temperature.every) == (0.4, 7.0) and a3.q_temperature is None and a0.taps == 0
    l1, r1 = p1.left, p1.right
    assert (p1.kind, p1.combine, p1.left_norm, p1.right_norm) == ("mixer_pair", "normed_mean", "l1.mix.left.out", "l1.mix.right.out")
    assert (l1.num_heads, l1.num_kv_heads, l1.head_dim, l1.value_dim, l1.scale, l1.taps) == (4, 2, 12, 14, 0.3, 3)
    assert (l1.norm_scope, l1.rot_pairs, l1.position.dims, l1.position.base, l1.sink) == ("projection", "neighbours", 8, 777.0, "l1.mix.left.sink")
    assert l1.gate_weight is None and l1.q_bias is None and p2.left.taps == 1 and p2.left.position.dims == 0
    assert (r1.kind, r1.heads, r1.dim, r1.vdim, r1.decay, r1.eps) == ("lightning_attention", 3, 10, 6, (0.5, 0.97, 0.9995), 1e-5)
    f0, f1 = spec.layers[0].feed_forward, spec.layers[1].feed_forward
    assert (f0.kind, f0.activation, f0.intermediate) == ("gated_mlp", "silu", 44) and spec.layers[2].feed_forward is None
    assert (f1.experts, f1.top, f1.intermediate, f1.score, f1.normalize, f1.weigh, f1.activation, f1.gate_weights) == \
        (5, 2, 22, "sigmoid", False, "input", "relu_squared", ())


def test_what_a_request_keeps():
    from llmengine.engine.model import Model
    from llmengine.parts.base import BuildEnv, KVNeed
    m = Model(describe_kasarax(KasaraxConfig.from_dict(KASARAX_A)), BuildEnv(torch.device("cpu"), torch.float32, CpuOps(), 4))
    assert m.windows == [0] and m.portion_multiple == 1 and m.capturable
    kinds = [[type(n) is KVNeed or n.name for n in needs] for needs in m.run_needs]
    assert kinds == [[True], [True, "gated_attention.conv", "lightning.state"], [True, "lightning.state"], [True]]  # one tap keeps nothing
    assert m.run_needs[1][1].shape == (2, 4 * 12 + 2 * 12 + 2 * 14)


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][0]["mixer"].update(heads=5), "multiple of kv_heads"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(heads=5), "multiple of kv_heads"),
    (lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(dims=7), "even"),
    (lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(dims=14), "at most dim"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(conv=0), "at least one tap"),
    (lambda c: c["layers"][1]["mixer"]["right"].update(decay=[0.5, 0.9]), "a number a head"),
    (lambda c: c["layers"][1]["mixer"]["right"].update(decay=0.5), "must be a list"),
    (lambda c: c["layers"][1]["mixer"]["right"]["decay"].__setitem__(1, 1.01), "lies in [0, 1]"),
    (lambda c: c["layers"][1]["mixer"].pop("right"), "right"),
    (lambda c: c["layers"][0]["mixer"]["q_temp"].update(every=0), "every must be positive"),
    (lambda c: c["layers"][0]["mixer"]["q_temp"].pop("coef"), "coef"),
    (lambda c: c["layers"][0].update(type="conv"), "unknown layer type"),
    (lambda c: c["layers"][0]["mlp"].update(kind="sparse"), "unknown kind"),
    (lambda c: c["layers"][0]["mlp"].update(ff=0), "ff must be positive"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=6), "6 of 5 experts"),
    (lambda c: c.pop("width"), "width"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c.update(layers=[]), "non-empty"),
])
def test_configuration_errors(change, message):
    cfg = copy.deepcopy(KASARAX_A)
    change(cfg)
    with pytest.raises(ConfigError) as e:
        KasaraxConfig.from_dict(cfg)
    assert message in str(e.value)


@pytest.mark.parametrize("name", sorted(KASARAX))
def test_sizes_that_only_tensor_shapes_give(name, tmp_path):
    full = KASARAX[name][0]
    write_model(str(tmp_path / "m"), full, torch.float32)
    parsed = config_from_dir(str(tmp_path / "m"))[1]
    assert parsed == KasaraxConfig.from_dict(full)
    cfg = copy.deepcopy(full)
    del cfg["vocab"], cfg["width"]
    for l in cfg["layers"]:
        for m in ([l["mixer"]] if l["type"] == "attention" else [l["mixer"]["left"], l["mixer"]["right"]]):
            for key in ("heads", "kv_heads", "dim", "vdim", "conv"):
                m.pop(key, None)
        if l["mlp"] and l["mlp"]["kind"] == "dense":
            del l["mlp"]["ff"]
        elif l["mlp"]:
            del l["mlp"]["expert"]["ff"], l["mlp"]["router"]["experts"]
    with open(tmp_path / "m" / "config.json", "w") as f:
        json.dump(cfg, f)
    assert config_from_dir(str(tmp_path / "m"))[1] == parsed
    assert sizes_from_tensors(full, lambda n: (1, 1))["layers"] == full["layers"]   # what the file says stays


def test_random_weights_mode(tmp_path):
    d = llmengine.write_random_model(str(tmp_path / "m"), KASARAX_B, seed=3, dtype=torch.bfloat16)
    arch, parsed = config_from_dir(d)
    assert arch.name == "Kasarax" and len(parsed.layers) == 5
    names = set(P.read_safetensors(str(tmp_path / "m" / "model.safetensors")))
    assert names >= {"embed", "final.norm", "l0.mix.left.v.conv", "l0.mix.right.out", "l2.mix.o.b", "l2.mlp.e3.down", "l1.mlp.router"}
    assert not names & {"l0.norm2", "l1.mlp.e0.gate", "l2.mix.sink", "l0.mix.left.g", "l1.mlp.correction"}


# ---------------------------------------------------------------------------------------------- the plain rules by hand
def test_plain_denominator_by_hand():
    p = P.softmax_with_term(torch.tensor([0.0, 1.0], dtype=torch.float64), torch.tensor(0.0, dtype=torch.float64))
    assert math.isclose(float(p[0]), 1 / (2 + math.e)) and math.isclose(float(p[1]), math.e / (2 + math.e))
    p = P.softmax_with_term(torch.tensor([3.0], dtype=torch.float64), torch.tensor(5.0, dtype=torch.float64))
    assert math.isclose(float(p[0]), math.exp(3) / (math.exp(3) + math.exp(5)))


def test_plain_query_temperature_by_hand_and_the_table():
    t = {"coef": 0.5, "every": 4}
    assert [P.query_temperature(p, t) for p in (0, 2)] == [1.0, 1.0]
    assert math.isclose(P.query_temperature(3, t), 1 + 0.5 * math.log(2)) and math.isclose(P.query_temperature(6, t), 1 + 0.5 * math.log(2))
    assert math.isclose(P.query_temperature(7, t), 1 + 0.5 * math.log(3)) and P.query_temperature(7, None) == 1.0
    for coef, every in ((0.3, 7), (1.7, 1), (0.0, 5), (0.25, 2.5)):
        table = query_temperatures(QueryTemperatureSpec(coef, every, 300))
        want = np.array([P.query_temperature(p, {"coef": coef, "every": every}) for p in range(300)])
        assert table.dtype == np.float32 and np.abs(table - want).max() < 1e-6


def test_plain_convolution_by_hand():
    st, w = {}, torch.tensor([[1.0, 10.0, 100.0]], dtype=torch.float64)
    y = P.short_conv(torch.tensor([[1.0], [2.0]], dtype=torch.float64), w, st, "c")
    assert y[:, 0].tolist() == [100.0, 210.0]                    # zeros before the sequence; the last tap meets the token itself
    assert P.short_conv(torch.tensor([[3.0]], dtype=torch.float64), w, st, "c")[0, 0] == 1 + 20 + 300


def test_plain_lightning_step_by_hand():
    S = torch.tensor([[[2.0], [4.0]]], dtype=torch.float64)
    k, q = torch.tensor([[1.0, 0.0]], dtype=torch.float64), torch.tensor([[1.0, 10.0]], dtype=torch.float64)
    S2, o = P.lightning_step(S, q, k, torch.tensor([[5.0]], dtype=torch.float64), torch.tensor([0.5], dtype=torch.float64))
    assert S2[0, :, 0].tolist() == [6.0, 2.0] and o[0, 0] == 26.0   # the read sees the write


def test_plain_weights_enter_before_the_activation():
    """One expert of one number: relu(up * s * h)^2 * down, s the score, and not s * relu(up * h)^2 * down."""
    w = {"router": torch.tensor([[1.0], [-1.0]], dtype=torch.float64), "e0.up": torch.tensor([[2.0]], dtype=torch.float64),
         "e0.down": torch.tensor([[3.0]], dtype=torch.float64), "e1.up": torch.tensor([[-5.0]], dtype=torch.float64), "e1.down": torch.tensor([[7.0]], dtype=torch.float64)}
    f = {"router": {"experts": 2, "top": 1}}
    h = torch.tensor([[0.5], [-0.25]], dtype=torch.float64)
    y = P.experts_ff(h, w, "", f)
    s0, s1 = 1 / (1 + math.exp(-0.5)), 1 / (1 + math.exp(-0.25))
    assert math.isclose(float(y[0, 0]), 3.0 * (2.0 * s0 * 0.5) ** 2) and math.isclose(float(y[1, 0]), 7.0 * (5.0 * s1 * 0.25) ** 2)


@pytest.mark.parametrize("name", sorted(KASARAX))
def test_plain_whole_against_portions_and_single_tokens(name):
    cfg = KASARAX[name][0]
    w = {k: v.double() for k, v in make_tensors(cfg, 2, torch.float32).items()}
    ids = random_ids(45, cfg["vocab"], 7)
    want = P.forward(cfg, w, ids)
    m = P.Plain(cfg, w)
    got = torch.cat([m.run(ids[a:b]) for a, b in ((0, 1), (1, 3), (3, 20), (20, 21), (21, 45))])
    assert float((got - want).abs().max()) < 1e-9


def test_every_tensor_matters():
    """Doubling (and shifting) any one tensor moves the plain logits by much more than the engine's tests allow."""
    for name in sorted(KASARAX):
        cfg = KASARAX[name][0]
        w = {k: v.double() for k, v in make_tensors(cfg, 2, torch.float32).items()}
        ids = random_ids(24, cfg["vocab"], 3)
        want = P.forward(cfg, w, ids)
        for k in w:
            other = dict(w)
            other[k] = w[k] * 1.5 + 0.3
            assert float((P.forward(cfg, other, ids) - want).abs().max()) > 3e-3, (name, k)


# ---------------------------------------------------------------------------------------------- the parts' own refusals
def test_options_that_do_not_go_together():
    from dataclasses import replace
    from llmengine.parts import build_part
    from llmengine.parts.base import BuildEnv
    env = BuildEnv(torch.device("cpu"), torch.float32, CpuOps(), 4)
    spec = describe_kasarax(KasaraxConfig.from_dict(KASARAX_A))
    a, left, ff = spec.layers[0].mixer, spec.layers[1].mixer.left, spec.layers[1].feed_forward
    for bad in (replace(a, unit_rms=True), replace(a, keys_as_values=True, value_dim=18), replace(a, value_mix="first"), replace(a, sink="s"),
                replace(left, q_conv=None), replace(left, own_kv=False, k_norm=None), replace(left, unit_rms=True, q_norm=None, k_norm=None)):
        with pytest.raises(ValueError):
            build_part("mixer", bad, env)
    for bad in (replace(ff, activation="silu"), replace(ff, identity=1), replace(ff, weigh="both"), replace(ff, gate_weights=ff.up_weights, activation="silu"),
                replace(ff, gate_weights=ff.up_weights[:2])):
        with pytest.raises(ValueError):
            build_part("feed_forward", bad, env)


# ---------------------------------------------------------------------------------------------- the engine's host side
@pytest.fixture(scope="module", params=["ka", "kc"])
def cpu_engine(request, tmp_path_factory):
    """The engine on the test double of the kernels: batch building, block tables, state slots, the wiring of the parts."""
    cfg, page = KASARAX[request.param]
    d = write_model(str(tmp_path_factory.mktemp("kasarax_" + request.param)), cfg, torch.float32, sharp=True)
    eng = llmengine.Engine(d, "fp32", device="cpu", ops=CpuOps(), block_size=page, num_blocks=40)
    eng.configure_cache(num_blocks=40, block_size=page, num_slots=3)
    return eng, P.read_model(d), cfg


def far(got, want):
    return float(np.abs(np.asarray(got) - np.asarray(want)).max()) / max(1.0, float(np.abs(np.asarray(want)).max()))


def test_engine_on_the_test_double_matches_plain(cpu_engine):
    eng, (pc, pw), cfg = cpu_engine
    a, b = random_ids(37, cfg["vocab"], 1), random_ids(11, cfg["vocab"], 2)
    want = {k: P.forward(pc, pw, ids).numpy() for k, ids in (("a", a), ("b", b))}
    got = eng.run_step([(1, a, list(range(len(a))))], end=[1]).numpy()
    assert far(got, want["a"]) < 1e-4
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
        assert far(row, ref[pos]) < 1e-4, (rid, pos)
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
        assert far(a.double(), b) < 1e-4, r


def test_generation_through_the_scheduler_matches_plain(cpu_engine):
    eng, (pc, pw), cfg = cpu_engine
    prompt = random_ids(9, cfg["vocab"], 3)
    out, reason = eng.generate(prompt, 7)
    assert reason == "length" and out == P.greedy(pc, pw, prompt, 7)


def test_command_line_random_weights_mode(tmp_path):
    from test_cli import run_cli
    cfg = tmp_path / "c.json"
    cfg.write_text(json.dumps(KASARAX_B))
    out = tmp_path / "model"
    r = run_cli("--random-weights", str(out), "--config", str(cfg), "--seed", "4", "--dtype", "bf16")
    assert r.returncode == 0, r.stderr
    arch, parsed = config_from_dir(str(out))
    assert arch.name == "Kasarax" and len(parsed.layers) == 5
