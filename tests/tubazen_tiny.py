"""Small Tubazen configurations, random model folders in the design's own tensor names, and the comparison of the
engine with the plain implementation (tests/plain/tubazen_plain.py)."""
import json
import os

import torch
from safetensors.torch import save_file

from plain import tubazen_plain as TP


def left(heads, kv_heads, dim, vdim=None, rows=12, far=40, temp=(0.4, 16), scale=None):
    """``rows`` travels in the configuration for the maker of random tensors; a folder's config.json is without it."""
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim if vdim is None else vdim, "bias_rows": rows,
            "bias_max": far, "q_temp": {"coef": temp[0], "every": temp[1]}, "scale": dim ** -0.5 if scale is None else scale}


def right(heads, dim, rank):
    return {"heads": heads, "dim": dim, "decay_rank": rank}


def parallel(lm, rm, ff=None, ls=1.0, rs=1.0):
    return {"type": "parallel", "mixer": {"left": lm, "right": rm, "left_scale": ls, "right_scale": rs}, "mlp": dense(ff)}


def gla(heads, dim, vdim, tau, rank, ff=None):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau, "decay_rank": rank}, "mlp": dense(ff)}


def dense(ff):
    return None if ff is None else {"kind": "dense", "ff": ff}


def config(vocab, width, layers, eps=1e-6, logit_scale=1.5, positions=1024):
    return {"architecture": "Tubazen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": logit_scale,
            "max_positions": positions, "layers": layers}


# Sizes differ from one another wherever the design lets them: query and key heads, groups of one and of several, key and
# value heads, heads of the two mixers, ranks, few buckets and many, far distances below, at and above a page, both
# multipliers, layers without a feed-forward in the middle and last, both mixers first and last.
MIXED = config(101, 64, [
    parallel(left(4, 2, 16, 24, rows=12, far=40), right(3, 16, 8), 40, 0.8, 1.3),
    gla(3, 16, 24, 4.0, 8, 56),
    gla(2, 24, 8, 1.0, 12),
    parallel(left(3, 3, 32, rows=20, far=130, temp=(0.2, 50)), right(1, 32, 24), None, 1.1, 0.9),
    parallel(left(6, 3, 24, 16, rows=7, far=64, temp=(-0.2, 7), scale=0.4), right(2, 24, 16), 48, 1.4, 0.7),
    gla(1, 40, 64, 16.0, 4),
], eps=1e-5)
ONLY_LEFT = config(64, 48, [parallel(left(4, 2, 16, 8), right(1, 8, 8), None, 1.7, 0.0),
                            parallel(left(2, 1, 24, rows=30, far=64, temp=(0.5, 3)), right(1, 8, 8), None, 1.2, 0.0)])
ONLY_RIGHT = config(64, 48, [parallel(left(1, 1, 8), right(3, 20, 8), None, 0.0, 1.5),
                             parallel(left(1, 1, 8), right(2, 16, 16), None, 0.0, 0.8)])
ONLY_GLA = config(64, 48, [gla(3, 20, 12, 8.0, 8), gla(2, 16, 32, 1.0, 16)])
ONLY_DENSE = config(64, 48, [gla(1, 8, 8, 1.0, 8, 56), gla(1, 8, 8, 2.0, 8, 24)], logit_scale=1.0)
# sizes the vector and tensor-core forms take, sequences across several pages
WIDE = config(128, 128, [
    parallel(left(4, 2, 64, rows=32, far=200), right(2, 64, 32), 96, 1.3, 0.8),
    gla(2, 64, 128, 8.0, 16, 160),
    parallel(left(8, 2, 128, 64, rows=64, far=350), right(1, 128, 16), 96, 0.9, 1.4),
    gla(1, 128, 128, 16.0, 64),
    parallel(left(2, 1, 48, rows=16, far=65), right(1, 256, 16), 64),
    gla(2, 256, 32, 4.0, 8, 64),
    parallel(left(4, 4, 96, rows=10, far=33), right(4, 32, 16), None, 1.1, 1.0),
])
# sizes that are multiples of nothing: every vectorized or tensor-core form refuses them
ODD = config(77, 50, [
    parallel(left(3, 1, 10, 14, rows=9, far=21), right(3, 7, 5), 22),
    gla(3, 7, 11, 3.0, 5, 30),
    parallel(left(5, 5, 12, 9, rows=5, far=100), right(1, 36, 3), 26, 1.2, 0.8),
    gla(1, 33, 27, 5.0, 9),
    parallel(left(6, 2, 14, 6, rows=2, far=17), right(2, 33, 9), None, 0.7, 1.1),
], eps=1e-4, logit_scale=0.8)
CONFIGS = {"mixed": (MIXED, 1), "left": (ONLY_LEFT, 2), "right": (ONLY_RIGHT, 3), "gla": (ONLY_GLA, 4),
           "dense": (ONLY_DENSE, 5), "wide": (WIDE, 6), "odd": (ODD, 7)}


def random_config(rng, nice):
    """A configuration drawn with ``rng`` (random.Random): 2 to 5 layers, sizes that the vector and tensor-core forms
    take (``nice``) or that are multiples of nothing."""
    pick = rng.choice
    width = pick([64, 128, 192, 256]) if nice else pick([50, 72, 100, 136])
    layers = []
    for _ in range(rng.randrange(2, 6)):
        ff = pick([None, 64, 128, 256]) if nice else pick([None, 30, 52, 100])
        if rng.random() < 0.4:
            layers.append(gla(pick([1, 2, 4]), pick([16, 32, 64, 128]) if nice else pick([8, 20, 33, 40]),
                              pick([16, 32, 64, 128]) if nice else pick([8, 12, 27, 40]), pick([1.0, 4.0, 16.0]),
                              pick([8, 16, 64]) if nice else pick([3, 5, 12]), ff))
            continue
        kv = pick([1, 2, 3])
        dim, vdim = pick([(32, 32), (48, 48), (64, 64), (96, 96), (128, 64), (64, 128)]) if nice else \
            (pick([8, 12, 24, 40, 72]), pick([8, 12, 20, 40, 56]))
        rows = pick([2, 5, 8, 16, 32, 40])
        lm = left(kv * pick([1, 2, 4]), kv, dim, vdim, rows=rows, far=rows // 2 + pick([1, 20, 64, 150]),
                  temp=(pick([0.1, 0.5]), pick([5, 64, 100])), scale=pick([None, 0.1]))
        rm = right(pick([1, 2, 4]), pick([16, 32, 64, 128]) if nice else pick([8, 20, 33, 40]),
                   pick([8, 16, 64]) if nice else pick([3, 5, 12]))
        layers.append(parallel(lm, rm, ff, pick([0.7, 1.0, 1.3]), pick([0.8, 1.0, 1.4])))
    return config(rng.randrange(90, 500), width, layers, eps=pick([1e-6, 1e-5]), logit_scale=pick([0.7, 1.0, 2.5]))


def random_tensors(cfg, seed, std=0.15):
    """Every tensor of a model file, by the design's names.  Nothing is left where it would hide a fault: norm weights
    around one and slopes that bend, biases away from zero, distance biases that decide between keys, decays that neither
    keep everything nor forget at once and that depend on the input, gates of either sign, weights of the earlier layers'
    outputs that matter."""
    g = torch.Generator().manual_seed(seed)
    d = cfg["width"]
    unit = std * (48.0 / d) ** 0.5           # results of the size they have at width 48, whatever the width
    out = {}

    def mat(name, *shape, s=unit, mean=0.0):
        out[name] = (mean + torch.randn(*shape, generator=g) * s).bfloat16()

    def norm(name):
        mat(name, d, s=0.3, mean=1.0)
        mat(name + ".b", d, s=0.2)
        out[name + ".alpha"] = (0.5 + 0.4 * torch.rand((), generator=g)).bfloat16()

    def gate(name):
        mat(name, d, d, s=2 * unit)
        mat(name + ".b", d, s=0.7, mean=0.5)

    mat("embed", cfg["vocab"], d, s=1.0)
    mat("pos", cfg["max_positions"], d, s=0.6)
    norm("embed.norm")
    mat("head", cfg["vocab"], d)
    norm("final.norm")
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        norm(p + "norm1")
        gate(p + "rg1")
        mat(p + "dwa", i + 2, s=0.25)
        out[p + "dwa"][-1] += 0.9
        if l["type"] == "gla":
            hk, hv = m["heads"] * m["dim"], m["heads"] * m["vdim"]
            for c, n in (("q", hk), ("k", hk), ("v", hv), ("g", hv)):
                mat(p + "mix." + c, n, d, s=2 * unit)
            mat(p + "mix.a1", m["decay_rank"], d, s=2 * unit)
            mat(p + "mix.a2", hk, m["decay_rank"], s=1.5 * m["decay_rank"] ** -0.5)
            mat(p + "mix.a2.b", hk, s=1.0, mean=1.5)
            mat(p + "mix.norm", m["vdim"], s=0.3, mean=1.0)
            mat(p + "mix.o", d, hv, s=std * (48.0 / hv) ** 0.5)
        else:
            a, r = m["left"], m["right"]
            hq, hk, hv, ho = a["heads"] * a["dim"], a["kv_heads"] * a["dim"], a["kv_heads"] * a["vdim"], a["heads"] * a["vdim"]
            q = p + "mix.left."
            for c, n in (("q", hq), ("k", hk), ("v", hv)):
                mat(q + c, n, d, s=2 * unit)
                mat(q + c + ".b", n, s=0.5)
            mat(q + "rel", a["bias_rows"], a["heads"], s=1.5)
            mat(q + "g", ho, d, s=2 * unit)
            mat(q + "o", d, ho, s=std * (48.0 / ho) ** 0.5)
            mat(q + "o.b", d, s=0.3)
            hd, q = r["heads"] * r["dim"], p + "mix.right."
            for c in "rkvga":
                mat(q + c, hd, d, s=2 * unit)
            mat(q + "a.b", hd, s=1.0)
            mat(q + "w1", r["decay_rank"], d, s=2 * unit)
            mat(q + "w2", hd, r["decay_rank"], s=2.0 * r["decay_rank"] ** -0.5)
            mat(q + "w0", hd, s=1.5, mean=-2.0)
            mat(q + "norm", hd, s=0.3, mean=1.0)
            mat(q + "o", d, hd, s=std * (48.0 / hd) ** 0.5)
        if l["mlp"]:
            norm(p + "norm2")
            gate(p + "rg2")
            ff = l["mlp"]["ff"]
            mat(p + "mlp.gate", ff, d, s=2 * unit)
            mat(p + "mlp.up", ff, d, s=2 * unit)
            mat(p + "mlp.down", d, ff, s=std * (48.0 / ff) ** 0.5)
    return out


def without_ranks(cfg):
    """What a model folder's config.json holds: ranks and buckets are only in the tensors' shapes."""
    cfg = json.loads(json.dumps(cfg))
    for l in cfg["layers"]:
        if l["type"] == "gla":
            l["mixer"].pop("decay_rank")
        else:
            l["mixer"]["right"].pop("decay_rank")
            l["mixer"]["left"].pop("bias_rows")
    return cfg


def make_folder(tmp, name, tensors_edit=None, cfg=None, seed=None):
    if cfg is None:
        cfg, seed = CONFIGS[name]
    folder = os.path.join(str(tmp), "tubazen_" + name)
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
        ref = TP.forward(cfg, tensors, tokens)
        top = max(top, float(ref.abs().max()))
        diffs += [(float((torch.as_tensor(row).double() - ref[p]).abs().max()), i, p) for p, row in sorted(got_rows.items())]
        if dtype != "float32":
            lost += (TP.forward(cfg, tensors, tokens, store=as_bfloat16) - ref).abs().max(dim=1).values.tolist()
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
