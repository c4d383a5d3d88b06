"""The Fofapel design without a GPU: its configuration, model spec and tensor plan, and the plain implementation's
own invariants."""
import copy
import math
import random

import pytest
import torch

import fofapel_tiny as T
from plain import fofapel_plain as FP

D = torch.float64


def _typed(cfg):
    from transformer_b200.api import _typed
    return _typed(cfg)


def _tensors(cfg, seed):
    return {k: v.double() if v.is_floating_point() else v for k, v in T.random_tensors(cfg, seed).items()}


def test_configuration_reads_every_size_and_round_trips():
    arch, meta = _typed(T.MIXED)
    assert arch.name == "fofapel"
    assert len(meta.layers) == 6 and meta.eps == 1e-5 and meta.vocab == 101 and meta.width == 64 and meta.alpha == 2.0
    a = meta.layers[0].mixer.left
    assert (a.heads, a.kv_heads, a.dim, a.window, a.rot_dims, a.rot_base, a.scale) == (4, 2, 16, 21, 8, 10000.0, 0.5)
    assert meta.layers[2].mixer.left.rot_dims == 0 and meta.layers[2].mixer.left.window == 0
    r = meta.layers[0].mixer.right
    assert (r.heads, r.dim, r.decay_rank) == (3, 16, 8)
    assert (meta.layers[0].mixer.left_scale, meta.layers[0].mixer.right_scale) == (0.8, 1.3)
    f = meta.layers[0].mlp
    assert (f.expert.ff, f.expert.limit, f.experts, f.top, f.shared.ff, f.shared.limit) == (24, 1.0, 5, 2, 40, 2.0)
    assert meta.layers[1].mlp.ff == 40 and meta.layers[2].mlp is None and meta.layers[3].mlp.shared is None
    assert type(meta).from_dict(meta.to_dict()) == meta


def test_the_rank_of_the_decay_comes_from_the_tensors():
    from transformer_b200.config.registry import ConfigError
    arch, meta = _typed(T.without_ranks(T.MIXED))
    with pytest.raises(ConfigError):
        arch.build_spec(meta)
    shapes = {n: tuple(t.shape) for n, t in T.random_tensors(*T.CONFIGS["mixed"]).items()}
    assert arch.refine(meta, shapes) == _typed(T.MIXED)[1]


def test_model_spec():
    arch, meta = _typed(T.MIXED)
    spec = arch.build_spec(meta)
    spec.validate()
    assert all(l.arrangement == "post_norm" and l.mixer.kind == "side_by_side" for l in spec.layers)
    kinds = [None if l.feed_forward is None else l.feed_forward.kind for l in spec.layers]
    assert kinds == ["moe", "swiglu", None, "moe", "moe", "swiglu"]
    m = dict(spec.layers[0].mixer.params)
    left, right = dict(m["left"].params), dict(m["right"].params)
    assert left["values"] == "keys" and left["sink_value"] == 0.0 and left["out_scale"] == 0.8 and left["window"] == 21
    assert right["out_scale"] == 1.3 and right["rank"] == 8
    assert dict(spec.layers[0].mixer_norm.params)["stream"] == 2.0 and "stream" not in dict(spec.final_norm.params)


@pytest.mark.parametrize("bad", [
    lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3),
    lambda c: c["layers"][0]["mixer"]["left"].update(vdim=8),
    lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=18),
    lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(size=0),
    lambda c: c["layers"][0]["mixer"].pop("right"),
    lambda c: c["layers"][0]["mixer"]["right"].update(heads=0),
    lambda c: c["layers"][0]["mlp"]["router"].update(top=6),
    lambda c: c["layers"][0]["mlp"]["expert"].pop("limit"),
    lambda c: c["layers"][0]["mlp"]["shared"].update(limit=0),
    lambda c: c["layers"][0].update(type="attention"),
    lambda c: c["layers"][1]["mlp"].update(kind="glu"),
    lambda c: c.pop("postln_alpha"),
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
    from transformer_b200.weights.loader import check_rules
    cfg, seed = T.CONFIGS[name]
    arch, meta = _typed(cfg)
    present = {n: (tuple(t.shape), "I32" if t.dtype == torch.int32 else "BF16") for n, t in T.random_tensors(cfg, seed).items()}
    chosen = check_rules(arch.tensor_plan(meta), present, name)
    assert all(v is not None for v in chosen.values())


def test_random_model_folder_has_the_design_s_tensor_names(tmp_path):
    import transformer_b200 as tb
    from transformer_b200.weights.loader import check_rules, open_tensors
    for cfg in (T.MIXED, T.random_config(random.Random(5), True), T.random_config(random.Random(6), False)):
        folder = tb.write_random_model(str(tmp_path / f"m{cfg['width']}_{cfg['vocab']}"), cfg, seed=1)
        arch, meta = _typed(cfg)
        files = open_tensors(folder)
        check_rules(arch.tensor_plan(meta), {n: files.shape_dtype(n) for n in files.names()}, folder)
        read, tensors = FP.read_folder(folder)
        assert _typed(read)[1] == meta
        for n, t in tensors.items():
            if n.endswith(".table"):        # the experts of a token differ, and all of them are there
                E = next(l["mlp"]["router"]["experts"] for i, l in enumerate(cfg["layers"]) if n.startswith(f"l{i}."))
                assert t.dtype == torch.int32 and int(t.min()) >= 0 and int(t.max()) < E
                assert all(len(set(row)) == len(row) for row in t.tolist())
        assert FP.forward(read, tensors, [1, 2, 3]).shape == (3, cfg["vocab"])


# ---- the plain implementation --------------------------------------------------------------------------------------
def test_plain_small_parts():
    g = torch.Generator().manual_seed(0)
    x, w, b = (torch.randn(4, 10, generator=g, dtype=D) for _ in range(3))
    ref = torch.nn.functional.layer_norm(x, (10,), w[0], b[0], 1e-3)
    assert float((FP.layer_norm(x, w[0], b[0], 1e-3) - ref).abs().max()) < 1e-12
    assert float((FP.gelu_tanh(x) - torch.nn.functional.gelu(x, approximate="tanh")).abs().max()) < 1e-12
    s = torch.tensor([0.5, -1.0, 2.0], dtype=D)
    full = torch.softmax(torch.cat([s, torch.zeros(1, dtype=D)]), 0)
    assert float((FP.softmax_off_by_one(s) - full[:3]).abs().max()) < 1e-12
    assert float(FP.softmax_off_by_one(s - 200.0).sum()) < 1e-80 and float(FP.softmax_off_by_one(s + 200.0).sum()) > 1 - 1e-12
    assert list(FP.visible(9, 4)) == [6, 7, 8, 9] and list(FP.visible(2, 4)) == [0, 1, 2] and len(FP.visible(9, None)) == 10


def test_plain_rotation_of_adjacent_pairs():
    v = torch.arange(10, dtype=D)
    r = FP.rotate_pairs(v, 3, 6, 100.0)
    assert torch.equal(r[6:], v[6:])
    for i in range(3):
        z = complex(v[2 * i], v[2 * i + 1]) * complex(math.cos(3 * 100.0 ** (-2 * i / 6)), math.sin(3 * 100.0 ** (-2 * i / 6)))
        assert abs(float(r[2 * i]) - z.real) < 1e-12 and abs(float(r[2 * i + 1]) - z.imag) < 1e-12
    # scores depend on the distance alone, and a turned head is as long as before
    q, k = torch.randn(8, dtype=D), torch.randn(8, dtype=D)
    s1 = FP.rotate_pairs(q, 9, 8, 100.0) @ FP.rotate_pairs(k, 4, 8, 100.0)
    s2 = FP.rotate_pairs(q, 25, 8, 100.0) @ FP.rotate_pairs(k, 20, 8, 100.0)
    assert abs(float(s1 - s2)) < 1e-12 and abs(float(FP.rotate_pairs(q, 9, 8, 100.0).norm() - q.norm())) < 1e-12


def test_plain_recurrence_writes_fades_and_adds_its_bonus():
    """One head of two key channels: a value written at token 0 is read at token 2 faded by the decays of token 1 alone
    (a token's decay acts after its own read), and the token itself counts with the bonus and not with the state."""
    r, k = torch.zeros(3, 1, 2, dtype=D), torch.zeros(3, 1, 2, dtype=D)
    v = torch.zeros(3, 1, 2, dtype=D)
    dec = torch.tensor([[[0.5, 0.1]], [[0.25, 0.2]], [[0.3, 0.3]]], dtype=D)
    u = torch.tensor([[3.0, 7.0]], dtype=D)
    k[0, 0, 0], v[0, 0] = 2.0, torch.tensor([1.0, -1.0], dtype=D)
    r[2, 0, 0], r[0, 0, 0], r[1, 0, 0] = 1.0, 1.0, 1.0
    o = FP.recurrence(r, k, v, dec, u)
    assert torch.allclose(o[0, 0], 3.0 * 2.0 * v[0, 0])        # bonus, the state is still empty
    assert torch.allclose(o[1, 0], 2.0 * v[0, 0])              # written undiminished
    assert torch.allclose(o[2, 0], 0.25 * 2.0 * v[0, 0])       # faded by token 1
    # against the closed form
    g = torch.Generator().manual_seed(2)
    r, k, v = (torch.randn(7, 2, 3, generator=g, dtype=D) for _ in range(3))
    dec, u = torch.rand(7, 2, 3, generator=g, dtype=D), torch.randn(2, 3, generator=g, dtype=D)
    o = FP.recurrence(r, k, v, dec, u)
    for t in range(7):
        for h in range(2):
            want = (r[t, h] * u[h] * k[t, h]).sum() * v[t, h]
            for j in range(t):
                fade = torch.ones(3, dtype=D)
                for s in range(j + 1, t):
                    fade = fade * dec[s, h]
                want = want + (r[t, h] * fade * k[j, h]).sum() * v[j, h]
            assert torch.allclose(o[t, h], want)


def test_plain_token_shift_and_table_of_experts():
    h = torch.tensor([[1.0, 2.0], [3.0, 5.0]], dtype=D)
    mu = torch.tensor([0.25, 1.0], dtype=D)
    assert torch.equal(FP.token_shift(h, mu), torch.tensor([[0.75, 0.0], [2.5, 2.0]], dtype=D))
    cfg, seed = T.CONFIGS["shared"]
    w = FP.sub(_tensors(cfg, seed), "l0.mlp.")
    f = cfg["layers"][0]["mlp"]
    x = torch.randn(3, cfg["width"], generator=torch.Generator().manual_seed(1), dtype=D)
    toks = [5, 9, 5]
    out = FP.table_experts(x, toks, w, f)
    for t, tok in enumerate(toks):
        want = torch.zeros(cfg["width"], dtype=D)
        for e in w["table"][tok].tolist():
            g, u = x[t] @ w[f"e{e}.gate"].T, x[t] @ w[f"e{e}.up"].T
            g, u = torch.minimum(g, torch.tensor(1.0, dtype=D)), torch.clamp(u, -1.0, 1.0)
            want += (g / (1 + torch.exp(-1.702 * g)) * (u + 1)) @ w[f"e{e}.down"].T / 3
        g, u = torch.clamp(x[t] @ w["shared.gate"].T, max=2.0), torch.clamp(x[t] @ w["shared.up"].T, -2.0, 2.0)
        want += torch.sigmoid(w["shared.sg"][0] @ x[t]) * ((g / (1 + torch.exp(-1.702 * g)) * (u + 1)) @ w["shared.down"].T)
        assert float((out[t] - want).abs().max()) < 1e-12


def test_plain_later_tokens_do_not_change_earlier_logits():
    cfg, seed = T.CONFIGS["mixed"]
    t = _tensors(cfg, seed)
    a = FP.forward(cfg, t, [5, 9, 33, 2, 71, 8, 8, 40])
    b = FP.forward(cfg, t, [5, 9, 33, 2, 71, 1, 2, 3])
    assert float((a[:5] - b[:5]).abs().max()) < 1e-12 and float((a[5:] - b[5:]).abs().max()) > 1e-3


@pytest.mark.parametrize("name, edit", [
    ("left", lambda t, c: t.update({k: torch.zeros_like(v) for k, v in t.items() if k.endswith("left.q.b")})),
    ("left", lambda t, c: t.update({k: torch.zeros_like(v) for k, v in t.items() if k.endswith("left.k.b")})),
    ("left", lambda t, c: t.update({k: torch.zeros_like(v) for k, v in t.items() if k.endswith("left.g")})),
    ("left", lambda t, c: [l["mixer"]["left"]["mask"].update(size=l["mixer"]["left"]["mask"]["size"] + 1) for l in c["layers"]]),
    ("left", lambda t, c: [l["mixer"]["left"].update(rot={"base": 100.0, "dims": 8}) for l in c["layers"]]),
    ("right", lambda t, c: t.update({k: torch.zeros_like(v) for k, v in t.items() if k.endswith("right.u")})),
    ("right", lambda t, c: t.update({k: torch.zeros_like(v) for k, v in t.items() if k.endswith("right.w2")})),
    ("right", lambda t, c: t.update({k: torch.full_like(v, 5.0) for k, v in t.items() if k.endswith("right.w0")})),
    ("right", lambda t, c: t.update({k: torch.zeros_like(v) for k, v in t.items() if ".mu." in k})),
    ("shared", lambda t, c: t.update({"l0.mlp.shared.sg": torch.zeros_like(t["l0.mlp.shared.sg"])})),
    ("shared", lambda t, c: t.update({"l0.mlp.table": (t["l0.mlp.table"] + 1) % 6})),
    ("shared", lambda t, c: c["layers"][0]["mlp"]["shared"].update(limit=1.0)),
    ("experts", lambda t, c: c["layers"][0]["mlp"]["expert"].update(limit=1.3)),
    ("dense", lambda t, c: t.update({"l0.norm2.b": torch.zeros_like(t["l0.norm2.b"])})),
    ("dense", lambda t, c: c.update(postln_alpha=1.0)),
])
def test_mechanisms_left_out_would_show(name, edit):
    """The test weights are made so that every mechanism matters: the plain implementation with one of them changed
    moves the logits beyond what the engine is held to in float32, and mostly far beyond the bfloat16 rule."""
    cfg, seed = T.CONFIGS[name]
    t = _tensors(cfg, seed)
    tokens = torch.randint(0, cfg["vocab"], (90,), generator=torch.Generator().manual_seed(3)).tolist()
    ref = FP.forward(cfg, t, tokens)
    t, cfg = dict(t), copy.deepcopy(cfg)
    edit(t, cfg)
    moved = (FP.forward(cfg, t, tokens) - ref).abs().max(dim=1).values
    assert float(moved.max()) > 50 * T.FP32_TOL, f"moved by {float(moved.max()):.2e}"
