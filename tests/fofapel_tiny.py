"""Small Fofapel configurations, random model folders in the design's own tensor names, and the comparison of the
engine with the plain implementation (tests/plain/fofapel_plain.py)."""
import json
import os

import torch
from safetensors.torch import save_file

from plain import fofapel_plain as FP


def left(heads, kv_heads, dim, window=None, dims=None, base=10000.0, scale=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": 2.0 * dim ** -0.5 if scale is None else scale}
    if window is not None:
        m["mask"] = {"size": window}
    if dims != 0:
        m["rot"] = {"base": base, "dims": dim if dims is None else dims}
    return m


def right(heads, dim, rank):
    """``rank`` travels in the configuration for the maker of random tensors; a folder's config.json is without it."""
    return {"heads": heads, "dim": dim, "decay_rank": rank}


def layer(lm, rm, mlp, ls=1.0, rs=1.0):
    return {"type": "parallel", "mixer": {"left": lm, "right": rm, "left_scale": ls, "right_scale": rs}, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, limit=1.0, shared=None, shared_limit=2.0):
    f = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    if shared is not None:
        f["shared"] = {"ff": shared, "limit": shared_limit}
    return f


def config(vocab, width, layers, eps=1e-6, alpha=2.0):
    return {"architecture": "Fofapel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "postln_alpha": alpha,
            "max_context": 1024, "layers": layers}


# Sizes differ from one another wherever the design lets them: query and key heads, groups of one and of several,
# heads of the two mixers, ranks, a rotation of a part of the head, of all of it and of none, windows below, at and
# above a page and none, both multipliers, one to three experts per token, with a shared expert and without, layers
# without a feed-forward, every kind of feed-forward first and last.
MIXED = config(101, 64, [
    layer(left(4, 2, 16, window=21, dims=8), right(3, 16, 8), moe(24, 5, 2, shared=40), 0.8, 1.3),
    layer(left(6, 3, 24, window=64, scale=0.4), right(2, 24, 16), dense(40), 1.4, 0.7),
    layer(left(3, 3, 32, dims=0), right(1, 32, 24), None, 1.1, 0.9),
    layer(left(4, 1, 8, window=100, base=500.0), right(4, 8, 8), moe(16, 3, 3, limit=0.7), 0.6, 1.2),
    layer(left(2, 2, 16, window=1), right(2, 40, 12), moe(32, 4, 1, shared=24, shared_limit=0.8)),
    layer(left(8, 2, 16, window=65, dims=4), right(2, 16, 8), dense(48), 1.2, 1.2),
], eps=1e-5)
ONLY_LEFT = config(64, 48, [layer(left(4, 2, 16, window=30, dims=8), right(1, 8, 8), None, 1.7, 0.0),
                            layer(left(2, 1, 24, window=70), right(1, 8, 8), None, 1.2, 0.0)])
ONLY_RIGHT = config(64, 48, [layer(left(1, 1, 8, window=4), right(3, 20, 8), None, 0.0, 1.5),
                             layer(left(1, 1, 8, window=4), right(2, 16, 16), None, 0.0, 0.8)])
ONLY_DENSE = config(64, 48, [layer(left(1, 1, 8, window=4), right(1, 8, 8), dense(56))], alpha=0.7)
ONLY_EXPERTS = config(64, 48, [layer(left(1, 1, 8, window=4), right(1, 8, 8), moe(24, 6, 2))])
ONLY_SHARED = config(64, 48, [layer(left(1, 1, 8, window=4), right(1, 8, 8), moe(24, 6, 3, shared=32))], alpha=1.0)
# sizes the vector and tensor-core forms take, sequences across several pages
WIDE = config(128, 128, [
    layer(left(4, 2, 64, window=90), right(2, 64, 32), moe(64, 8, 2, shared=96), 1.3, 0.8),
    layer(left(8, 2, 32, window=128, dims=16, base=5e5), right(1, 128, 64), dense(96), 0.9, 1.4),
    layer(left(2, 1, 128, window=200), right(1, 256, 16), moe(64, 8, 1)),
    layer(left(4, 4, 96, window=33), right(4, 32, 16), None, 1.1, 1.0),
], alpha=2.0)
# sizes that are multiples of nothing: every vectorized or tensor-core form refuses them
ODD = config(77, 50, [
    layer(left(3, 1, 10, window=19, dims=6), right(3, 7, 5), moe(9, 3, 2, shared=11)),
    layer(left(5, 5, 12), right(1, 36, 3), dense(22), 1.2, 0.8),
    layer(left(6, 2, 14, window=40, dims=2), right(2, 33, 9), moe(7, 2, 1, limit=0.5)),
], eps=1e-4, alpha=1.2)
CONFIGS = {"mixed": (MIXED, 1), "left": (ONLY_LEFT, 2), "right": (ONLY_RIGHT, 3), "dense": (ONLY_DENSE, 4),
           "experts": (ONLY_EXPERTS, 5), "shared": (ONLY_SHARED, 6), "wide": (WIDE, 7), "odd": (ODD, 8)}


def random_config(rng, nice):
    """A configuration drawn with ``rng`` (random.Random): 2 to 5 layers, sizes that the vector and tensor-core forms
    take (``nice``) or that are multiples of nothing."""
    pick = rng.choice
    width = pick([64, 128, 256, 320]) if nice else pick([50, 72, 100, 136])
    layers = []
    for _ in range(rng.randrange(2, 6)):
        kv = pick([1, 2, 3])
        dim = pick([32, 48, 64, 96, 128]) if nice else pick([8, 12, 24, 40, 72])
        lm = left(kv * pick([1, 2, 4]), kv, dim, window=pick([None, 1, 16, 63, 64, 65, 150]),
                  dims=pick([0, dim, dim // 2, dim]) // 2 * 2, base=pick([10000.0, 500000.0, 100.0]),
                  scale=pick([None, 0.2, 0.4]))
        rm = right(pick([1, 2, 4]), pick([16, 32, 64, 128]) if nice else pick([8, 20, 33, 40]),
                   pick([8, 16, 64]) if nice else pick([3, 5, 12]))
        r = rng.random()
        if r < 0.15:
            mlp = None
        elif r < 0.45:
            mlp = dense(pick([64, 128, 320]) if nice else pick([30, 52, 100]))
        else:
            e = pick([2, 4, 8, 16]) if nice else pick([3, 5, 7])
            mlp = moe(pick([32, 64, 128]) if nice else pick([12, 20, 44]), e, rng.randrange(1, min(e, 4) + 1),
                      limit=pick([0.5, 1.5, 7.0]), shared=pick([None, 64, 96]) if nice else pick([None, 21, 30]),
                      shared_limit=pick([0.5, 3.0]))
        layers.append(layer(lm, rm, mlp, pick([0.7, 1.0, 1.3]), pick([0.8, 1.0, 1.4])))
    return config(rng.randrange(90, 700), width, layers, eps=pick([1e-6, 1e-5]), alpha=pick([0.8, 1.0, 2.5]))


def random_tensors(cfg, seed, std=0.15):
    """Every tensor of a model file, by the design's names.  Nothing is left where it would hide a fault: norm weights
    around one, biases away from zero, mixes between none and all of the token before, decays that neither keep
    everything nor forget at once and that depend on the input, a bonus of the size of what the memory holds, gates of
    either sign, pairs that reach their limits."""
    g = torch.Generator().manual_seed(seed)
    d = cfg["width"]
    unit = std * (48.0 / d) ** 0.5           # results of the size they have at width 48, whatever the width
    out = {}

    def mat(name, *shape, s=unit):
        out[name] = (torch.randn(*shape, generator=g) * s).bfloat16()

    def around_one(name, n, spread=0.3):
        out[name] = (1.0 + spread * torch.randn(n, generator=g)).bfloat16()

    def norm(name):
        around_one(name, d)
        mat(name + ".b", d, s=0.3)

    mat("embed", cfg["vocab"], d, s=1.0)
    mat("head", cfg["vocab"], d)
    norm("final.norm")
    for i, l in enumerate(cfg["layers"]):
        p, a, r, f = f"l{i}.", l["mixer"]["left"], l["mixer"]["right"], l["mlp"]
        norm(p + "norm1")
        hq, hk = a["heads"] * a["dim"], a["kv_heads"] * a["dim"]
        mat(p + "mix.left.q", hq, d, s=2 * unit)
        mat(p + "mix.left.k", hk, d, s=2 * unit)
        mat(p + "mix.left.q.b", hq, s=0.5)
        mat(p + "mix.left.k.b", hk, s=0.5)
        mat(p + "mix.left.g", a["heads"], d, s=3 * unit)
        mat(p + "mix.left.o", d, hq, s=std * (48.0 / hq) ** 0.5)
        hd = r["heads"] * r["dim"]
        for c in "rkvgw":
            out[p + f"mix.right.mu.{c}"] = torch.rand(d, generator=g).bfloat16()
        for c in "rkvg":
            mat(p + f"mix.right.{c}", hd, d, s=2 * unit)
        mat(p + "mix.right.w1", r["decay_rank"], d, s=2 * unit)
        mat(p + "mix.right.w2", hd, r["decay_rank"], s=2.0 * r["decay_rank"] ** -0.5)
        out[p + "mix.right.w0"] = (torch.rand(hd, generator=g) * 4.0 - 4.0).bfloat16()
        mat(p + "mix.right.u", r["heads"], r["dim"], s=0.7)
        around_one(p + "mix.right.norm", hd)
        mat(p + "mix.right.o", d, hd, s=std * (48.0 / hd) ** 0.5)
        if not f:
            continue
        norm(p + "norm2")

        def pair(name, ff):
            mat(p + name + ".gate", ff, d, s=2 * unit)
            mat(p + name + ".up", ff, d, s=2 * unit)
            mat(p + name + ".down", d, ff, s=std * (48.0 / ff) ** 0.5)

        if f["kind"] == "dense":
            pair("mlp", f["ff"])
            continue
        E, top = f["router"]["experts"], f["router"]["top"]
        for e in range(E):
            pair(f"mlp.e{e}", f["expert"]["ff"])
        out[p + "mlp.table"] = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(cfg["vocab"])]).to(torch.int32)
        if f.get("shared"):
            pair("mlp.shared", f["shared"]["ff"])
            mat(p + "mlp.shared.sg", 1, d, s=3 * unit)
    return out


def without_ranks(cfg):
    """What a model folder's config.json holds: the ranks are only in the tensors' shapes."""
    cfg = json.loads(json.dumps(cfg))
    for l in cfg["layers"]:
        l["mixer"]["right"].pop("decay_rank")
    return cfg


def make_folder(tmp, name, tensors_edit=None, cfg=None, seed=None):
    if cfg is None:
        cfg, seed = CONFIGS[name]
    folder = os.path.join(str(tmp), "fofapel_" + name)
    if not os.path.isdir(folder):
        os.makedirs(folder)
        tensors = random_tensors(cfg, seed)
        if tensors_edit:
            tensors_edit(tensors)
        with open(os.path.join(folder, "config.json"), "w") as f:
            json.dump(without_ranks(cfg), f)
        save_file({k: v.contiguous() for k, v in tensors.items()}, os.path.join(folder, "model.safetensors"))
    return folder


FP32_TOL = 1e-4           # on logits of order one to ten
# bfloat16: against the plain implementation run exactly, measured in what that implementation itself loses when it
# rounds where a 16-bit path stores an activation: the mean over a request's positions and any single position.
BF16_MEAN, BF16_EACH = 1.5, 2.5
BF16_REL_TOL = 2.0 ** -5  # for comparisons of the engine with itself, of the largest |logit|


def as_bfloat16(x):
    return x.bfloat16().to(x.dtype)


def check_requests(cfg, tensors, requests, dtype, label=""):
    """requests: [(tokens, {position: logits row of the engine})], held to the rules together (a request of a few tokens
    alone says little about what rounding costs the model)."""
    diffs, lost, top = [], [], 0.0
    for i, (tokens, got_rows) in enumerate(requests):
        ref = FP.forward(cfg, tensors, tokens)
        top = max(top, float(ref.abs().max()))
        diffs += [(float((torch.as_tensor(row).double() - ref[p]).abs().max()), i, p) for p, row in sorted(got_rows.items())]
        if dtype != "float32":
            lost += (FP.forward(cfg, tensors, tokens, store=as_bfloat16) - ref).abs().max(dim=1).values.tolist()
    if dtype == "float32":
        tol = FP32_TOL * max(1.0, top / 10.0)
    else:
        tol, rule = BF16_EACH * max(lost), BF16_MEAN * sum(lost) / len(lost)
        mean = sum(v for v, _, _ in diffs) / len(diffs)
        if len(diffs) >= 20:
            assert mean <= rule, f"{label}: mean |diff| {mean:.3e} > {rule:.3e}"
    for v, i, p in diffs:
        assert v <= tol, f"{label}: request {i}, position {p} (the first wrong one): |diff| {v:.3e} > {tol:.3e}"


def check_request(cfg, tensors, tokens, got_rows, dtype, label=""):
    check_requests(cfg, tensors, [(tokens, got_rows)], dtype, label)


def run_cuts(engine, tokens, cuts, graphs=False):
    """One request through the engine in steps of the given sizes (the rest one token at a time); returns
    {position: logits} for every position."""
    engine.use_graphs = graphs
    slot = engine.open()
    rows, at = {}, 0
    for n in list(cuts) + [1] * (len(tokens) - sum(cuts)):
        lg = engine.step([slot], [tokens[at:at + n]], [list(range(n))]).cpu()
        for i in range(n):
            rows[at + i] = lg[i].clone()
        at += n
    engine.close(slot)
    engine.check_kernels()
    return rows
