"""The Tubazen design without a GPU: its configuration, model spec and tensor plan, and the plain implementation's
own invariants."""
import copy
import math
import random
from fractions import Fraction

import pytest
import torch

import tubazen_tiny as T
from plain import tubazen_plain as TP

D = torch.float64


def _typed(cfg):
    from transformer_b200.api import _typed
    return _typed(cfg)


def _tensors(cfg, seed):
    return {k: v.double() for k, v in T.random_tensors(cfg, seed).items()}


def test_configuration_reads_every_size_and_round_trips():
    arch, meta = _typed(T.MIXED)
    assert arch.name == "tubazen"
    assert len(meta.layers) == 6 and meta.eps == 1e-5 and meta.vocab == 101 and meta.width == 64
    assert meta.logit_scale == 1.5 and meta.max_positions == 1024
    m = meta.layers[0].mixer
    a, r = m.left, m.right
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.bias_max, a.temp_coef, a.temp_every, a.bias_rows) == \
        (4, 2, 16, 24, 0.25, 40, 0.4, 16, 12)
    assert (r.heads, r.dim, r.decay_rank, m.left_scale, m.right_scale) == (3, 16, 8, 0.8, 1.3)
    x = meta.layers[1].mixer
    assert (x.heads, x.dim, x.vdim, x.tau, x.decay_rank) == (3, 16, 24, 4.0, 8)
    assert [l.ff for l in meta.layers] == [40, 56, None, None, 48, None]
    assert type(meta).from_dict(meta.to_dict()) == meta


def test_ranks_and_buckets_come_from_the_tensors():
    from transformer_b200.config.registry import ConfigError
    arch, meta = _typed(T.without_ranks(T.MIXED))
    with pytest.raises(ConfigError):
        arch.build_spec(meta)
    shapes = {n: tuple(t.shape) for n, t in T.random_tensors(*T.CONFIGS["mixed"]).items()}
    assert arch.refine(meta, shapes) == _typed(T.MIXED)[1]
    with pytest.raises(ConfigError):        # more buckets than the far distance allows
        arch.refine(meta, dict(shapes, **{"l0.mix.left.rel": (80, 4)}))


def test_model_spec():
    arch, meta = _typed(T.MIXED)
    spec = arch.build_spec(meta)
    spec.validate()
    assert spec.max_context == 1024
    assert [l.mixer.kind for l in spec.layers] == ["side_by_side", "gated_linear", "gated_linear", "side_by_side",
                                                   "side_by_side", "gated_linear"]
    assert all(l.arrangement == "pre_norm" and l.mixer_norm.kind == "tanh_norm" for l in spec.layers)
    assert [l.feed_forward is None for l in spec.layers] == [False, False, True, True, False, True]
    assert [len(l.extra) for l in spec.layers] == [2, 2, 1, 1, 2, 1]
    assert [e.joint for e in spec.order] == [None, 0, 1, 2, 3, 4] and spec.last_joint == 5
    assert [j.get()["terms"] for j in spec.joints] == [2, 3, 4, 5, 6, 7]
    left = dict(dict(spec.layers[0].mixer.params)["left"].params)
    assert left["distance_bias"] == (12, 40) and left["query_temp"] == (0.4, 16) and left["out_scale"] == 0.8
    assert dict(dict(spec.layers[0].mixer.params)["right"].params)["out_scale"] == 1.3


@pytest.mark.parametrize("bad", [
    lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3),
    lambda c: c["layers"][0]["mixer"]["left"].update(bias_max=6),
    lambda c: c["layers"][0]["mixer"]["left"].pop("bias_max"),
    lambda c: c["layers"][0]["mixer"]["left"]["q_temp"].update(every=0),
    lambda c: c["layers"][0]["mixer"]["left"]["q_temp"].pop("coef"),
    lambda c: c["layers"][0]["mixer"].pop("right"),
    lambda c: c["layers"][0]["mixer"]["right"].update(heads=0),
    lambda c: c["layers"][1]["mixer"].update(tau=0),
    lambda c: c["layers"][1]["mixer"].pop("tau"),
    lambda c: c["layers"][1]["mixer"].update(vdim=-1),
    lambda c: c["layers"][0].update(type="attention"),
    lambda c: c["layers"][1]["mlp"].update(kind="moe"),
    lambda c: c.pop("max_positions"),
    lambda c: c["norm"].pop("eps"),
])
def test_configuration_errors_are_named(bad):
    from transformer_b200.config.registry import ConfigError
    cfg = copy.deepcopy(T.MIXED)
    bad(cfg)
    with pytest.raises(ConfigError):
        _typed(cfg)


@pytest.mark.parametrize("name", list(T.CONFIGS))
def test_tensor_plan_names_every_tensor_of_a_model_file(name):
    from transformer_b200.weights.loader import WeightError, check_rules
    cfg, seed = T.CONFIGS[name]
    arch, meta = _typed(cfg)
    present = {n: (tuple(t.shape), "BF16") for n, t in T.random_tensors(cfg, seed).items()}
    chosen = check_rules(arch.tensor_plan(meta), present, name)
    assert all(v is not None for v in chosen.values())
    if cfg["layers"][-1]["mlp"] is None:    # what belongs to a feed-forward may be there without one
        last, d = f"l{len(cfg['layers']) - 1}.", cfg["width"]
        more = {last + "norm2": (d,), last + "norm2.b": (d,), last + "norm2.alpha": (), last + "rg2": (d, d), last + "rg2.b": (d,)}
        check_rules(arch.tensor_plan(meta), dict(present, **{n: (s, "BF16") for n, s in more.items()}), name)
    with pytest.raises(WeightError):
        check_rules(arch.tensor_plan(meta), dict(present, stray=((3,), "BF16")), name)


def test_random_model_folder_has_the_design_s_tensor_names(tmp_path):
    import transformer_b200 as tb
    from transformer_b200.weights.loader import check_rules, open_tensors
    for cfg in (T.MIXED, T.random_config(random.Random(5), True), T.random_config(random.Random(6), False)):
        folder = tb.write_random_model(str(tmp_path / f"m{cfg['width']}_{cfg['vocab']}"), cfg, seed=1)
        arch, meta = _typed(cfg)
        files = open_tensors(folder)
        check_rules(arch.tensor_plan(meta), {n: files.shape_dtype(n) for n in files.names()}, folder)
        read, tensors = TP.read_folder(folder)
        assert _typed(read)[1] == meta
        assert TP.forward(read, tensors, [1, 2, 3]).shape == (3, cfg["vocab"])


def test_parts_that_do_not_go_together_are_refused():
    from transformer_b200.parts.base import MIXERS
    from transformer_b200.parts.block import build_layer
    from transformer_b200.parts.spec import LayerSpec, PartSpec
    cpu = torch.device("cpu")
    biased = PartSpec.of("attention", width=32, nh=2, nkvh=1, dh=16, out_bias=True)
    norm = PartSpec.of("rmsnorm", width=32, eps=1e-6)
    build_layer(LayerSpec(biased, None, norm), torch.float32, cpu)
    with pytest.raises(ValueError, match="output bias"):
        build_layer(LayerSpec(biased, None, norm, arrangement="parallel"), torch.float32, cpu)
    for bad in (dict(distance_bias=(8, 4)), dict(query_temp=(0.1, 8)), dict(bias=True, conv_taps=3),
                dict(distance_bias=(8, 40), values="keys")):
        with pytest.raises(ValueError):
            MIXERS.build(PartSpec.of("attention", width=32, nh=2, nkvh=1, dh=16, **bad), torch.float32, cpu)


# ---- distance buckets -----------------------------------------------------------------------------------------------
def _exact_bucket(n, rows, far):
    """By whole numbers alone: the largest k with (far / half)^k <= (n / half)^(rows - half)."""
    half = rows // 2
    if n < half:
        return n
    k, base, have = 0, Fraction(far, half), Fraction(n, half) ** (rows - half)
    while k < rows - half and base ** (k + 1) <= have:
        k += 1
    return min(rows - 1, half + k)


@pytest.mark.parametrize("rows, far", [(2, 9), (3, 5), (7, 64), (8, 64), (10, 160), (12, 40), (16, 128), (20, 160), (24, 97)])
def test_buckets_of_distances(rows, far):
    """The engine's table and the plain function against whole numbers, also where a bucket starts exactly at a power."""
    from transformer_b200.parts.attention import distance_bucket, distance_buckets
    table = distance_buckets(rows, far)
    assert table[-1] == rows - 1 and (len(table) == 1 or table[-2] < rows - 1) and len(table) <= far + 1
    for n in range(far + 3):
        want = _exact_bucket(n, rows, far)
        assert distance_bucket(n, rows, far) == TP.bucket(n, rows, far) == want, (n, want)
        assert table[min(n, len(table) - 1)] == want


# ---- the plain implementation --------------------------------------------------------------------------------------
def test_plain_small_parts():
    g = torch.Generator().manual_seed(0)
    x = torch.randn(4, 10, generator=g, dtype=D)
    assert float((TP.gelu_tanh(x) - torch.nn.functional.gelu(x, approximate="tanh")).abs().max()) < 1e-12
    w = {"n": torch.full((10,), 2.0, dtype=D), "n.b": torch.full((10,), 0.5, dtype=D), "n.alpha": torch.tensor(0.3, dtype=D)}
    e = torch.exp(2 * 0.3 * x)
    assert float((TP.tanh_norm(x, w, "n") - (2 * (e - 1) / (e + 1) + 0.5)).abs().max()) < 1e-12
    hist = [torch.full((2, 3), v, dtype=D) for v in (1.0, 10.0, 100.0)]
    assert torch.equal(TP.depth_average(hist, torch.tensor([3.0, 2.0, 1.0], dtype=D)), torch.full((2, 3), 123.0, dtype=D))
    gw = {"r": torch.eye(3, dtype=D), "r.b": torch.tensor([0.0, 1.0, -1.0], dtype=D)}
    got = TP.residual_gate(torch.tensor([[2.0, -1.0, 1.0]], dtype=D), gw, "r")
    assert torch.allclose(got, torch.tensor([[1 / (1 + math.exp(-2.0)), 0.5, 0.5]], dtype=D))


def test_plain_query_temperature_steps_at_multiples():
    assert [TP.query_temperature(p, 0.5, 4) for p in (0, 2)] == [1.0, 1.0]
    assert TP.query_temperature(3, 0.5, 4) == TP.query_temperature(6, 0.5, 4) == 1.0 + 0.5 * math.log(2.0)
    assert TP.query_temperature(7, 0.5, 4) == 1.0 + 0.5 * math.log(3.0)


def test_plain_gated_linear_attention_fades_and_counts_the_token_itself():
    g = torch.Generator().manual_seed(2)
    q, k = (torch.randn(7, 2, 3, generator=g, dtype=D) for _ in range(2))
    v, alpha = torch.randn(7, 2, 5, generator=g, dtype=D), torch.rand(7, 2, 3, generator=g, dtype=D)
    o = TP.gla_recurrence(q, k, v, alpha)
    for t in range(7):
        for h in range(2):
            want = torch.zeros(5, dtype=D)
            for j in range(t + 1):
                fade = torch.ones(3, dtype=D)
                for s in range(j + 1, t + 1):
                    fade = fade * alpha[s, h]
                want = want + (q[t, h] * fade * k[j, h]).sum() * v[j, h]
            assert torch.allclose(o[t, h], want)


def test_plain_delta_rule_removes_fades_and_writes():
    """One head: with a removal rate of one and no decay, writing under a unit key replaces what lay there; both terms
    read the old state; the key keeps its length where it is written."""
    e = torch.eye(3, dtype=D)
    k = torch.stack([2.0 * e[0], e[0], e[1]])[:, None]
    v = torch.tensor([[1.0, 2, 3], [4, 5, 6], [7, 8, 9]], dtype=D)[:, None]
    r, one = e[0].expand(3, 1, 3), torch.ones(3, 1, 3, dtype=D)
    o = TP.right_recurrence(r, one, k, v, one)
    assert torch.allclose(o[0, 0], 2 * v[0, 0], atol=1e-5)
    assert torch.allclose(o[1, 0], v[1, 0], atol=1e-5) and torch.allclose(o[2, 0], v[1, 0], atol=1e-5)
    half = one * 0.5            # decays to a half, removes another half of the OLD state: nothing is left of it
    o = TP.right_recurrence(r, half, k, v, half)
    assert torch.allclose(o[1, 0], v[1, 0], atol=1e-5)
    assert torch.allclose(o[2, 0], 0.5 * v[1, 0], atol=1e-5)


def test_plain_later_tokens_do_not_change_earlier_logits():
    cfg, seed = T.CONFIGS["mixed"]
    t = _tensors(cfg, seed)
    a = TP.forward(cfg, t, [5, 9, 33, 2, 71, 8, 8, 40])
    b = TP.forward(cfg, t, [5, 9, 33, 2, 71, 1, 2, 3])
    assert float((a[:5] - b[:5]).abs().max()) < 1e-12 and float((a[5:] - b[5:]).abs().max()) > 1e-3


def _zero(*ends):
    return lambda t, c: t.update({k: torch.zeros_like(v) for k, v in t.items() if k.endswith(ends)})


@pytest.mark.parametrize("name, edit", [
    ("left", _zero("left.q.b")), ("left", _zero("left.v.b")), ("left", _zero("left.o.b")),
    ("left", _zero("left.g")), ("left", _zero("left.rel")),
    ("left", lambda t, c: [l["mixer"]["left"].update(bias_max=l["mixer"]["left"]["bias_max"] + 8) for l in c["layers"]]),
    ("left", lambda t, c: [l["mixer"]["left"]["q_temp"].update(coef=0.0) for l in c["layers"]]),
    ("left", lambda t, c: [l["mixer"]["left"]["q_temp"].update(every=l["mixer"]["left"]["q_temp"]["every"] + 1) for l in c["layers"]]),
    ("right", _zero("right.a.b")), ("right", _zero("right.a")), ("right", _zero("right.w2")), ("right", _zero("right.w0")),
    ("right", _zero("right.g")),
    ("gla", _zero("mix.a2.b")), ("gla", _zero("mix.a1")), ("gla", _zero("mix.g")),
    ("gla", lambda t, c: c["layers"][0]["mixer"].update(tau=7.0)),
    ("dense", _zero("norm2.b")), ("dense", _zero("rg2.b")), ("dense", _zero("rg1")),
    ("dense", lambda t, c: t.update({"l1.dwa": t["l1.dwa"] * torch.tensor([0.0, 1.0, 1.0], dtype=D)})),
    ("dense", lambda t, c: t.update({"embed.norm.alpha": t["embed.norm.alpha"] * 1.2})),
    ("dense", _zero("pos")),
])
def test_mechanisms_left_out_would_show(name, edit):
    """The test weights are made so that every mechanism matters: the plain implementation with one of them changed
    moves the logits beyond what the engine is held to in float32, and mostly far beyond the bfloat16 rule.  (A bias on
    the keys alone changes no weight of a softmax without rotation: the kernel's own test looks at it in the cache.)"""
    cfg, seed = T.CONFIGS[name]
    t = _tensors(cfg, seed)
    tokens = torch.randint(0, cfg["vocab"], (90,), generator=torch.Generator().manual_seed(3)).tolist()
    ref = TP.forward(cfg, t, tokens)
    t, cfg = dict(t), copy.deepcopy(cfg)
    edit(t, cfg)
    moved = (TP.forward(cfg, t, tokens) - ref).abs().max(dim=1).values
    assert float(moved.max()) > 50 * T.FP32_TOL, f"moved by {float(moved.max()):.2e}"
