"""The Tubazen design in the engine against the plain implementation: each mechanism alone, prompts against decoding,
portions, unequal batches, reused slots and pages, the first tokens, far keys and buckets' edges, long decoding,
generation; and its kernels alone with inputs made so that a fault shows."""
import json
import math
import random
import subprocess
import sys

import pytest
import torch

import tubazen_tiny as T
from plain import tubazen_plain as TP
from tiny import ROOT, TraceRun, random_prompts

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    tmp = tmp_path_factory.mktemp("tubazen")
    return {name: T.make_folder(tmp, name) for name in T.CONFIGS}


def _load(folder, dtype, **kw):
    import transformer_b200 as tb
    kw.setdefault("max_tokens", 2048)
    return tb.load(folder, dtype=dtype, **kw)


def _tokens(folder, n, seed):
    cfg, _ = TP.read_folder(folder)
    return random_prompts(cfg["vocab"], [n], seed)[0]


def greedy(cfg, tensors, prompt, steps):
    seq, out = list(prompt), []
    for _ in range(steps):
        tok = int(torch.argmax(TP.forward(cfg, tensors, seq)[-1]))
        out.append(tok)
        seq.append(tok)
    return out


def _same(a, b, dtype, label):
    """Rows of two runs of the engine, within its rounding."""
    for p in a:
        if p in b:
            tol = 1e-4 if dtype == "float32" else 2 * T.BF16_REL_TOL * float(max(r.abs().max() for r in a.values()))
            assert float((a[p] - b[p]).abs().max()) <= tol, f"{label}: position {p}"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["left", "right", "gla", "dense"])
def test_each_mechanism_alone(name, dtype, folders):
    """One kind of part: every position of a prompt that crosses a page border, then six tokens decoded."""
    cfg, tensors = TP.read_folder(folders[name])
    tokens = _tokens(folders[name], 106, 11)
    rows = T.run_cuts(_load(folders[name], dtype), tokens, [100])
    T.check_request(cfg, tensors, tokens, rows, dtype, name)


@pytest.mark.parametrize("dtype", DTYPES)
def test_prompt_against_decoding_token_by_token(dtype, folders):
    cfg, tensors = TP.read_folder(folders["mixed"])
    tokens = _tokens(folders["mixed"], 110, 5)
    engine = _load(folders["mixed"], dtype)
    whole = T.run_cuts(engine, tokens, [110])
    single = T.run_cuts(engine, tokens, [])
    T.check_request(cfg, tensors, tokens, whole, dtype, "whole")
    T.check_request(cfg, tensors, tokens, single, dtype, "token by token")
    if dtype == "float32":
        _same(whole, single, dtype, "whole against single tokens")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cuts", [[2, 2, 3, 57, 64, 2], [63, 1, 64, 2], [5, 130], [128, 2, 2], [1, 1, 2, 100]])
def test_portions_of_a_prompt(cuts, dtype, folders):
    """A prompt fed in portions, down to two tokens, with cuts at and beside page borders and buckets' edges: the memories
    come from the step before, positions and distances go on."""
    cfg, tensors = TP.read_folder(folders["mixed"])
    tokens = _tokens(folders["mixed"], 140, 6)
    rows = T.run_cuts(_load(folders["mixed"], dtype), tokens, cuts)
    T.check_request(cfg, tensors, tokens, rows, dtype, f"cuts {cuts}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_step_cut_into_pieces_by_the_engine(dtype, folders):
    cfg, tensors = TP.read_folder(folders["mixed"])
    tokens = _tokens(folders["mixed"], 100, 16)
    rows = T.run_cuts(_load(folders["mixed"], dtype, max_step_tokens=37), tokens, [95])
    T.check_request(cfg, tensors, tokens, rows, dtype, "pieces")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_unequal_batch_equals_each_request_alone(name, dtype, folders):
    """Prompts of 1, 63, 64 and 130 tokens in one step, then decoded together while the short ones end; in slots
    and pages that an earlier batch has used."""
    cfg, tensors = TP.read_folder(folders[name])
    engine = _load(folders[name], dtype, max_tokens=640)
    engine.use_graphs = False
    lens, extra = [1, 63, 64, 130], [2, 6, 4, 8]
    seqs = [_tokens(folders[name], n + e, 20 + i) for i, (n, e) in enumerate(zip(lens, extra))]
    old = [engine.open() for _ in range(3)]
    engine.step(old, [_tokens(folders[name], n, 40 + n) for n in (100, 70, 129)])
    for s in old:
        engine.close(s)
    slots = [engine.open() for _ in seqs]
    rows = [dict() for _ in seqs]
    lg = engine.step(slots, [s[:n] for s, n in zip(seqs, lens)], [list(range(n)) for n in lens]).cpu()
    at = 0
    for i, n in enumerate(lens):
        for p in range(n):
            rows[i][p] = lg[at + p]
        at += n
    step = 0
    while True:
        live = [i for i in range(len(seqs)) if lens[i] + step < len(seqs[i])]
        if not live:
            break
        lg = engine.step([slots[i] for i in live], [[seqs[i][lens[i] + step]] for i in live]).cpu()
        for j, i in enumerate(live):
            rows[i][lens[i] + step] = lg[j]
        step += 1
    engine.check_kernels()
    alone = _load(folders[name], dtype)
    for i, seq in enumerate(seqs):
        T.check_request(cfg, tensors, seq, rows[i], dtype, f"request {i} in the batch")
        single = T.run_cuts(alone, seq, [lens[i]])
        if dtype == "float32":
            _same(single, rows[i], dtype, f"request {i} alone and in the batch")


def test_a_slot_and_its_pages_used_again_hold_nothing_of_their_past(folders):
    engine = _load(folders["mixed"], "float32", max_tokens=256)
    a, b = _tokens(folders["mixed"], 130, 1), _tokens(folders["mixed"], 70, 2)
    fresh = T.run_cuts(_load(folders["mixed"], "float32", max_tokens=256), b, [60])
    T.run_cuts(engine, a, [120])
    again = T.run_cuts(engine, b, [60])
    for p in fresh:
        assert torch.equal(fresh[p], again[p]), f"position {p}"


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_first_tokens_of_a_sequence(dtype, folders):
    """Sequences of one, two and three tokens side by side: one key in the softmax, empty memories, position zero."""
    cfg, tensors = TP.read_folder(folders["mixed"])
    engine = _load(folders["mixed"], dtype)
    seqs = [_tokens(folders["mixed"], n, 80 + n) for n in (1, 2, 3)]
    slots = [engine.open() for _ in seqs]
    lg = engine.step(slots, seqs, [list(range(len(s))) for s in seqs]).cpu()
    T.check_requests(cfg, tensors, [(seqs[0], {0: lg[0]}), (seqs[1], {0: lg[1], 1: lg[2]}),
                                    (seqs[2], {0: lg[3], 1: lg[4], 2: lg[5]})], dtype, "sequences of one to three")


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_through_graphs(dtype, folders):
    """Three prompt tokens, then 200 tokens decoded through the replayed step: distances pass every bucket, the query's
    multiplier grows, the memories are carried 200 times."""
    cfg, tensors = TP.read_folder(folders["mixed"])
    tokens = _tokens(folders["mixed"], 203, 9)
    engine = _load(folders["mixed"], dtype)
    assert engine.graph_safe
    slot = engine.open()
    rows = {2: engine.step([slot], [tokens[:3]]).cpu()[0]}
    for p in range(3, len(tokens)):
        rows[p] = engine.step([slot], [[tokens[p]]]).cpu()[0].clone()
    engine.check_kernels()
    assert engine._graphs, "the decode steps were not replayed from a graph"
    T.check_request(cfg, tensors, tokens, rows, dtype, "long decoding")


@pytest.mark.parametrize("dtype", DTYPES)
def test_many_sequences_decoded_together(dtype, folders):
    """More sequences than the few-token products take: 20 prompts of one to three tokens, then decoded together through
    the graph, against each alone."""
    engine = _load(folders["wide"], dtype, max_tokens=4096)
    seqs = [_tokens(folders["wide"], 1 + i % 3 + 5, 100 + i) for i in range(20)]
    slots = [engine.open() for _ in seqs]
    lens = [1 + i % 3 for i in range(20)]
    engine.step(slots, [s[:n] for s, n in zip(seqs, lens)])
    got = [dict() for _ in seqs]
    for j in range(5):
        lg = engine.step(slots, [[s[n + j]] for s, n in zip(seqs, lens)]).cpu()
        for i in range(20):
            got[i][lens[i] + j] = lg[i].clone()
    engine.check_kernels()
    cfg, tensors = TP.read_folder(folders["wide"])
    T.check_requests(cfg, tensors, list(zip(seqs, got)), dtype, "20 sequences")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name, n, cuts", [("wide", 420, [410]), ("wide", 300, [70, 200]), ("odd", 90, [66, 3])])
def test_sizes_that_reach_the_fast_kernels_and_sizes_that_none_takes(name, n, cuts, dtype, folders):
    cfg, tensors = TP.read_folder(folders[name])
    tokens = _tokens(folders[name], n, 3)
    rows = T.run_cuts(_load(folders[name], dtype), tokens, cuts)
    T.check_request(cfg, tensors, tokens, rows, dtype, name)


@pytest.mark.parametrize("seed", [0, 1, 2, 3, 4, 5])
def test_configurations_drawn_at_random(seed, tmp_path):
    """Layers and sizes drawn at random (two of three draws take sizes that reach the vector and tensor-core forms): a
    prompt across several pages and twelve decoded tokens."""
    rng = random.Random(3000 + seed)
    cfg = T.random_config(rng, nice=seed % 3 != 2)
    folder = T.make_folder(tmp_path, f"drawn{seed}", cfg=cfg, seed=seed)
    cfg, tensors = TP.read_folder(folder)
    n = rng.randrange(150, 280)
    tokens = random_prompts(cfg["vocab"], [n + 12], seed)[0]
    for dtype in DTYPES:
        rows = T.run_cuts(_load(folder, dtype), tokens, [n])
        T.check_request(cfg, tensors, tokens, rows, dtype, f"drawn {seed}")


def test_equal_layers_are_replayed_and_give_the_same(tmp_path):
    """Layers of equal parts are recorded once a step and replayed with their own tensors, among them the ones that the
    block leaves to the joint behind it; bit for bit what running each from Python gives."""
    cfg = T.config(64, 64, [T.parallel(T.left(2, 1, 16), T.right(2, 16, 8), 40, 0.9, 0.7)] * 3 + [T.gla(2, 16, 16, 2.0, 8)] * 2)
    folder = T.make_folder(tmp_path, "equal", cfg=cfg, seed=9)
    engine = _load(folder, "bfloat16")
    tokens = random_prompts(64, [90], 4)[0]
    both = []
    for tapes in (True, False):
        engine.use_tapes = tapes
        both.append(T.run_cuts(engine, tokens, [40, 45]))
    assert engine._tape_maps and all(m is not None for m in engine._tape_maps.values()), "nothing was replayed"
    for p in both[0]:
        assert torch.equal(both[0][p], both[1][p])
    cfg, tensors = TP.read_folder(folder)
    T.check_request(cfg, tensors, tokens, both[0], "bfloat16", "replayed")


def test_the_context_ends_with_the_position_table(tmp_path):
    import transformer_b200 as tb
    cfg = T.config(64, 48, [T.gla(2, 16, 16, 2.0, 8)], positions=20)
    engine = _load(T.make_folder(tmp_path, "short", cfg=cfg, seed=3), "float32")
    slot = engine.open()
    engine.step([slot], [list(range(19))])
    engine.step([slot], [[1]])
    with pytest.raises(tb.CacheError):
        engine.step([slot], [[2]])


def test_random_weights_on_the_device_equal_the_written_folder(tmp_path):
    import transformer_b200 as tb
    cfg = T.CONFIGS["mixed"][0]
    folder = tb.write_random_model(str(tmp_path / "written"), cfg, seed=5, std=0.1)
    tokens = random_prompts(cfg["vocab"], [70], 1)[0]
    a = tb.load(folder, dtype="bfloat16", max_tokens=512)
    b = tb.random_model(cfg, seed=5, dtype="bfloat16", max_tokens=512, std=0.1)
    la = a.step([a.open()], [tokens], [list(range(70))]).cpu()
    lb = b.step([b.open()], [tokens], [list(range(70))]).cpu()
    assert torch.equal(la, lb)


def test_greedy_generation_through_the_entry_point(folders):
    import transformer_b200 as tb
    cfg, tensors = TP.read_folder(folders["mixed"])
    prompts = [_tokens(folders["mixed"], n, 30 + n) for n in (7, 66, 2)]
    got = tb.generate(_load(folders["mixed"], "float32"), prompts, max_steps=6, stop_tokens=()).tokens
    assert got == [greedy(cfg, tensors, p, 6) for p in prompts]
    res = tb.generate(_load(folders["mixed"], "bfloat16"), prompts, max_steps=6, stop_tokens=())
    assert [len(t) for t in res.tokens] == [6, 6, 6]


def test_trace_runner_and_command_line(folders, tmp_path):
    cfg, tensors = TP.read_folder(folders["mixed"])
    a, b = _tokens(folders["mixed"], 70, 1), _tokens(folders["mixed"], 9, 2)
    run = TraceRun(folders["mixed"], "float32", str(tmp_path / "out"), 256, record_routing=False)
    run.step(0, [{"id": "a", "tokens": a[:66], "want": [0, 65]}, {"id": "b", "tokens": b[:8], "want": [7]}])
    run.step(1, [{"id": "a", "tokens": a[66:67], "want": [0]}, {"id": "b", "tokens": b[8:9], "want": []}], end=["b"])
    run.step(2, [{"id": "a", "tokens": a[67:68], "want": [0]}], end=["a"])
    first, second, third = (run.logits(i, cfg["vocab"]) for i in range(3))
    run.close()
    ref_a, ref_b = TP.forward(cfg, tensors, a), TP.forward(cfg, tensors, b)
    for got, want in ((first[0], ref_a[0]), (first[1], ref_a[65]), (first[2], ref_b[7]), (second[0], ref_a[66]),
                      (third[0], ref_a[67])):
        assert float((got.double() - want).abs().max()) <= T.FP32_TOL
    assert second.shape[0] == 1
    out = subprocess.run([sys.executable, "-m", "transformer_b200", "generate", "--model", folders["mixed"],
                          "--prompt", " ".join(map(str, b)), "--max-steps", "4", "--dtype", "float32", "--json"],
                         cwd=ROOT, capture_output=True, text=True, timeout=600)
    assert out.returncode == 0, out.stderr[-2000:]
    assert json.loads(out.stdout.strip().splitlines()[-1])["tokens"] == [greedy(cfg, tensors, b, 4)]


# ---- the mechanisms in other surroundings --------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
def test_gates_joints_and_biases_with_other_norms_and_parts(dtype):
    """Gated residuals, an average over the depth, an output bias, a linear memory and experts in pre-norm blocks with RMS
    norms, which take none of it in their own kernels: a prompt against single tokens, and the first token against the
    same sums in torch."""
    from transformer_b200.architectures.generic import plan_from_spec
    from transformer_b200.engine import Engine
    from transformer_b200.parts.spec import LayerSpec, ModelSpec, PartSpec, RunEntry
    from transformer_b200.weights.random_init import random_device_weights
    d, V, td = 64, 60, torch.float32 if dtype == "float32" else torch.bfloat16
    norm = PartSpec.of("rmsnorm", width=d, eps=1e-6)
    gate = PartSpec.of("sigmoid", width=d)
    att = PartSpec.of("attention", width=d, nh=4, nkvh=2, dh=16, bias=True, out_bias=True, out_scale=0.5, distance_bias=(8, 30),
                      position=PartSpec.of("rope", dh=16, theta=1e4, positions=256))
    gl = PartSpec.of("gated_linear", width=d, heads=2, dim=16, vdim=32, tau=2.0, rank=8, eps=1e-5, out_scale=1.5)
    sd = PartSpec.of("split_delta", width=d, heads=2, dim=32, rank=8, eps=1e-5)
    both = PartSpec.of("side_by_side", width=d, left=PartSpec.of("gated_linear", **dict(gl.params, out_scale=0.7)), right=att)
    moe = PartSpec.of("moe", width=d, di=48, nexp=4, nexp_use=2)
    dense = PartSpec.of("swiglu", width=d, di=40)
    layers = (LayerSpec(att, moe, norm, norm, extra=(("feed_forward_residual_gate", gate),)),
              LayerSpec(gl, dense, norm, norm, extra=(("mixer_residual_gate", gate),)),
              LayerSpec(sd, None, norm),
              LayerSpec(both, dense, norm, norm))
    spec = ModelSpec(width=d, vocab=V, max_context=256, layers=layers,
                     order=(RunEntry(0), RunEntry(1, joint=0), RunEntry(2, joint=1), RunEntry(3)),
                     joints=(PartSpec.of("depth_average", width=d, terms=2), PartSpec.of("depth_average", width=d, terms=3)),
                     embedding=PartSpec.of("positional_lookup", vocab=V, width=d, positions=256, scale=2.0), final_norm=norm,
                     head=PartSpec.of("linear", vocab=V, width=d, tied=False))
    dev = torch.device("cuda:0")
    weights = random_device_weights(plan_from_spec(spec), 3, td, dev, 0.3)
    engine = Engine(spec, weights, td, dev, max_tokens=512)
    tokens = random_prompts(V, [70], 1)[0]
    whole = engine.step([engine.open()], [tokens], [list(range(70))]).cpu()
    slot = engine.open()
    engine.step([slot], [tokens[:50]])
    tol = 1e-3 if dtype == "float32" else 0.06 * float(whole.abs().max())
    for p in range(50, 70):
        assert float((engine.step([slot], [[tokens[p]]]).cpu()[0] - whole[p]).abs().max()) < tol, p
    engine.check_kernels()
    if dtype == "bfloat16":
        return
    # a model of the first token alone, in torch: each sum as the block's words say
    W = {k: v.double().cpu() for k, v in weights.items()}
    part = lambda i, n: {k[3]: v for k, v in W.items() if k[:3] == ("layers", i, n)}
    rms = lambda x, w: x / torch.sqrt((x * x).mean() + 1e-6) * w
    x = W[("embedding", "table")][tokens[0]] * 2.0 + W[("embedding", "positions")][0]
    first = x
    m, h = part(0, "mixer"), rms(x, part(0, "mixer_norm")["weight"])
    v = (m["wqkv"] @ h + m["bqkv"])[96:].view(2, 16).repeat_interleave(2, 0).reshape(-1)        # one key: its value
    x = x + 0.5 * (m["wo"] @ v + m["bo"])
    f, h = part(0, "feed_forward"), rms(x, part(0, "feed_forward_norm")["weight"])
    top = torch.topk(f["router"] @ h, 2)
    y = sum(a * (f["wd"][e] @ (TP.silu(f["wgu"][e, :48] @ h) * (f["wgu"][e, 48:] @ h)))
            for a, e in zip(torch.softmax(top.values, 0), top.indices.tolist()))
    r = part(0, "feed_forward_residual_gate")
    x = x + y * torch.sigmoid(r["weight"] @ h + r["bias"])
    second = x
    x = W[("joints", 0, "weight")] @ torch.stack([first, x])
    m, h = part(1, "mixer"), rms(x, part(1, "mixer_norm")["weight"])
    z = (m["win"] @ h)
    q, k, v, g = z[:32].view(2, 16) / 4, z[32:64].view(2, 16), z[64:128].view(2, 32), z[128:]
    o = (q * k).sum(1, keepdim=True) * v
    o = (TP.rms(o, 1e-5) * m["norm"]).reshape(-1) * 1.5 * TP.silu(g)
    r = part(1, "mixer_residual_gate")
    x = x + (m["wo"] @ o) * torch.sigmoid(r["weight"] @ h + r["bias"])
    f, h = part(1, "feed_forward"), rms(x, part(1, "feed_forward_norm")["weight"])
    x = x + f["wd"] @ (TP.silu(f["wgu"][:40] @ h) * (f["wgu"][40:] @ h))
    x = W[("joints", 1, "weight")] @ torch.stack([first, second, x])
    seen = []

    class Stop(Exception):
        pass

    def stop(ctx, xx, pending, cache, state):
        from transformer_b200.parts.block import add_pending
        add_pending(ctx, xx, pending)
        seen.append(xx.cpu().double().clone())
        raise Stop
    engine.layers[2].forward, engine.use_tapes = stop, False
    slot = engine.open()
    with pytest.raises(Stop):
        engine.step([slot], [tokens[:3]])
    assert float((seen[0][0] - x).abs().max()) <= 1e-4 * max(1.0, float(x.abs().max()))


# ---- kernels alone, with inputs made so that a fault shows ---------------------------------------------------
def _td(dtype):
    return (torch.float32, "f32") if dtype == "float32" else (torch.bfloat16, "bf16")


def _ints(v):
    return torch.tensor(v, dtype=torch.int32, device="cuda")


class _Pages:
    """A batch of sequences over shuffled pages: lens_before tokens already there, lens_new in the step."""

    def __init__(self, lens_before, lens_new, g):
        self.before, self.new = lens_before, lens_new
        self.total = [a + b for a, b in zip(lens_before, lens_new)]
        n = sum((t + 63) // 64 for t in self.total) + 3
        perm = torch.randperm(n, generator=g).tolist()
        self.n_pages, self.max_pages = n, max((t + 63) // 64 for t in self.total)
        table = torch.zeros(len(lens_new), self.max_pages, dtype=torch.int32)
        for b, t in enumerate(self.total):
            for p in range((t + 63) // 64):
                table[b, p] = perm.pop()
        self.h_table, self.table = table, table.cuda()
        self.nt = sum(lens_new)
        starts = [0]
        for n_ in lens_new:
            starts.append(starts[-1] + n_)
        self.starts, self.seq_start = starts, _ints(starts)
        self.tok_seq = _ints([b for b, n_ in enumerate(lens_new) for _ in range(n_)])
        self.tok_pos = _ints([p for b, n_ in enumerate(lens_new) for p in range(lens_before[b], self.total[b])])

    def tiles(self, tq):
        rows = [(b, self.starts[b] + off, min(tq, n - off)) for b, n in enumerate(self.new) for off in range(0, n, tq)]
        return [_ints([r[i] for r in rows]) for i in range(3)] + [len(rows)]

    def put(self, cache, b, pos, rows):
        """rows [n, heads, dim] at positions pos, pos + 1, ... of sequence b."""
        for i, r in enumerate(rows):
            cache[self.h_table[b, (pos + i) // 64], :, (pos + i) % 64] = r


@pytest.mark.parametrize("kernel, dtype, splits", [("general", "float32", 1), ("general", "float32", 3), ("general", "bfloat16", 1),
                                                   ("mma", "bfloat16", 1), ("mma", "bfloat16", 3)])
@pytest.mark.parametrize("H, G, dk, dv, rows, far, window", [
    (4, 2, 64, 64, 12, 40, 1 << 30), (6, 2, 32, 32, 32, 130, 1 << 30), (2, 2, 128, 64, 8, 64, 1 << 30),
    (8, 1, 64, 128, 40, 300, 1 << 30), (3, 1, 96, 96, 2, 65, 1 << 30), (12, 1, 48, 48, 20, 11, 1 << 30), (4, 2, 64, 64, 16, 63, 96)])
def test_attention_with_a_bias_by_distance(kernel, dtype, splits, H, G, dk, dv, rows, far, window):
    """Every head's table favours, far above the rest, one bucket (its keys are then all that a query reads; a table or a
    distance that is one off reads others), the last bucket, the key itself, or nothing, with scores that ask for one key:
    prompts, portions and single tokens across pages, an output gate per entry, a multiplier and rows that are a part of
    wider ones whose other entries stay as they were."""
    from transformer_b200.csrc import lib
    from transformer_b200.parts.attention import distance_buckets
    td, sfx = _td(dtype)
    g = torch.Generator().manual_seed(H * dk + splits)
    pg = _Pages([0, 130, 64, 321, 40], [90, 1, 1, 1, 70], g)
    kc = torch.randn(pg.n_pages, G, 64, dk, generator=g).to(td)
    vc = torch.randn(pg.n_pages, G, 64, dv, generator=g).to(td)
    keys, vals = [], []
    for b, n in enumerate(pg.total):
        k = torch.randn(n, G, dk, generator=g)
        k, v = (k / k.norm(dim=-1, keepdim=True)).to(td), torch.randn(n, G, dv, generator=g).to(td)
        pg.put(kc, b, 0, k)
        pg.put(vc, b, 0, v)
        keys.append(k.double())
        vals.append(v.double())
    gz = (torch.randn(pg.nt, H * dv + 8, generator=g) * 2).to(td)
    ldo, scale, mult = H * dv + 8, 0.5, 1.25
    tq = lib.attention_window_mma_tile_tokens(H, G) if kernel == "mma" else lib.attention_tile_tokens(H, G)
    t_seq, t_t0, t_nq, count = pg.tiles(tq)
    at = torch.tensor(distance_buckets(rows, far))
    d_kc, d_vc, d_gz = kc.cuda(), vc.cuda(), gz.cuda()
    for which in ("one bucket", "last bucket", "itself", "one key"):
        rel = torch.randn(rows, H, generator=g) * 0.5
        if which == "one bucket":
            rel[torch.randint(0, rows, (H,), generator=g), torch.arange(H)] = 30.0
        elif which != "one key":
            rel[-1 if which == "last bucket" else 0] = 30.0
        q, want = torch.zeros(pg.nt, H, dk), torch.zeros(pg.nt, H, dv, dtype=torch.float64)
        for b in range(len(pg.new)):
            by = rel.double()[[TP.bucket(n, rows, far) for n in range(pg.total[b])]]
            for i in range(pg.new[b]):
                p, t = pg.before[b] + i, pg.starts[b] + i
                lo = max(0, p - window + 1)
                for h in range(H):
                    q[t, h] = torch.randn(dk, generator=g) * 4 if which != "one key" else \
                        keys[b][int(torch.randint(lo, p + 1, (1,), generator=g)), h // (H // G)].float() * 24.0
                qs = q[t].to(td).double()
                s = torch.einsum("jhc,hc->jh", keys[b][lo:p + 1].repeat_interleave(H // G, 1), qs) * scale
                w = torch.softmax(s + by[:p + 1 - lo].flip(0), 0)
                want[t] = torch.einsum("jh,jhc->hc", w, vals[b][lo:p + 1].repeat_interleave(H // G, 1))
        want *= torch.sigmoid(gz[:, 8:].double()).view(pg.nt, H, dv) * mult
        d_q, d_rel = q.to(td).cuda(), rel[at].t().contiguous().cuda()
        out = torch.full((pg.nt, ldo), 7.0, dtype=td, device="cuda")
        partial = torch.empty(pg.nt, H, splits, dv + 2, device="cuda")
        name = "tb_attention_window_mma_biased_bf16" if kernel == "mma" else "tb_attention_window_biased_" + sfx
        ok = lib.try_call(name, lib.ptr(d_q), lib.ptr(out), lib.ptr(d_kc), lib.ptr(d_vc), lib.ptr(d_gz[:, 8:]),
                          lib.ptr(t_seq), lib.ptr(t_t0), lib.ptr(t_nq), lib.ptr(pg.tok_pos), lib.ptr(pg.table),
                          lib.ptr(partial) if splits > 1 else 0, count, pg.nt, pg.max_pages, H * dk, H * dv + 8, H, G, dk, dv,
                          splits, window, 0, scale, 0.0, 0, 0, 0, mult, ldo, lib.ptr(d_rel), d_rel.shape[1] - 1)
        assert ok, "the kernel refused sizes it is meant to take"
        torch.cuda.synchronize()
        got = out.cpu()
        assert bool((got[:, H * dv:] == 7.0).all()), "entries beside the heads' were written"
        diff = (got[:, :H * dv].double().view(pg.nt, H, dv) - want).abs()
        assert float(diff.max()) <= (2e-5 if dtype == "float32" else 4e-2), f"{which}: {float(diff.max()):.3e}"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H, G, dk, dv, rdims, norm, lens", [(4, 2, 64, 32, 0, False, [70, 3]), (3, 1, 10, 7, 6, True, [5, 66]),
                                                            (6, 3, 24, 40, 8, True, [1, 1]), (2, 2, 16, 16, 0, False, [1, 2])])
def test_head_kernel_with_biases_and_a_multiplier_by_position(dtype, H, G, dk, dv, rdims, norm, lens):
    """Biases on queries, keys and values (before norm and rotation), the queries' multiplier at each position, every key
    and value in its row of its page and nowhere else."""
    from transformer_b200.csrc import lib
    from transformer_b200.parts.rope import Rope
    td, sfx = _td(dtype)
    g = torch.Generator().manual_seed(dk + H)
    pg = _Pages([62, 130], lens, g)
    wide = (H + G) * dk + G * dv
    ldz = wide + 8
    z = torch.randn(pg.nt, ldz, generator=g).to(td)
    bias, mult = torch.randn(wide, generator=g), torch.rand(256, generator=g) + 0.5
    qn, kn = torch.rand(H * dk, generator=g) + 0.5, torch.rand(G * dk, generator=g) + 0.5
    kc = torch.full((pg.n_pages, G, 64, dk), 9.0, dtype=td, device="cuda")
    vc = torch.full((pg.n_pages, G, 64, dv), 9.0, dtype=td, device="cuda")
    cos = sin = None
    if rdims:
        cos, sin = Rope({"dh": rdims, "theta": 100.0, "positions": 256}, td, torch.device("cuda")).tables()
    d_z, d_b, d_m, d_qn, d_kn = (t.cuda() for t in (z, bias, mult, qn, kn))
    lib.call("tb_qknorm_rope_cache_biased_" + sfx, lib.ptr(d_z), ldz, lib.ptr(d_b), lib.ptr(d_m), lib.ptr(d_qn) if norm else 0,
             lib.ptr(d_kn) if norm else 0, 1e-3, lib.ptr(pg.tok_seq), lib.ptr(pg.tok_pos), lib.ptr(pg.table), pg.max_pages,
             lib.ptr(cos), lib.ptr(sin), lib.ptr(kc), lib.ptr(vc), pg.nt, H, G, dk, dv, rdims, 0)
    torch.cuda.synchronize()

    def turned(x, p):
        y = x.clone()
        for i in range(rdims // 2):
            a = p * 100.0 ** (-2.0 * i / rdims)
            y[:, 2 * i] = x[:, 2 * i] * math.cos(a) - x[:, 2 * i + 1] * math.sin(a)
            y[:, 2 * i + 1] = x[:, 2 * i + 1] * math.cos(a) + x[:, 2 * i] * math.sin(a)
        return y
    u = z[:, :wide].double() + bias.double()
    want_k, want_v = torch.full(kc.shape, 9.0, dtype=torch.float64), torch.full(vc.shape, 9.0, dtype=torch.float64)
    tol = 2e-5 if dtype == "float32" else 4e-2
    for b, n in enumerate(pg.new):
        for i in range(n):
            t, p = pg.starts[b] + i, pg.before[b] + i
            q, k, v = u[t, :H * dk], u[t, H * dk:(H + G) * dk], u[t, (H + G) * dk:]
            if norm:
                q, k = TP.rms(q, 1e-3) * qn.double(), TP.rms(k, 1e-3) * kn.double()
            got = d_z[t, :H * dk].cpu().double().view(H, dk)
            assert float((got - turned(q.view(H, dk), p) * mult[p].double()).abs().max()) <= tol, f"query of token {t}"
            pg.put(want_k, b, p, [turned(k.view(G, dk), p)])
            pg.put(want_v, b, p, [v.view(G, dv)])
    assert float((kc.cpu().double() - want_k).abs().max()) <= tol
    assert float((vc.cpu().double() - want_v).abs().max()) <= tol


class _Memory:
    """A recurrence's kernels over a batch in slots, carried from step to step, beside the plain recurrence: what the
    kernels make of rows z = [.. | .. | v | gate] and of the decay's pre-activation, up to the gated heads."""

    def __init__(self, kind, dtype, H, dim, vdim, rank, seed):
        from transformer_b200.csrc import lib
        self.lib, (self.td, self.sfx), self.kind = lib, _td(dtype), kind
        self.H, self.dim, self.vdim, self.rank = H, dim, vdim, rank
        g = self.g = torch.Generator().manual_seed(seed)
        self.hk, self.hv = H * dim, H * vdim
        self.w2 = (torch.randn(self.hk, rank, generator=g) * 1.5 * rank ** -0.5).to(self.td)
        self.w0, self.ba = torch.randn(self.hk, generator=g), torch.randn(self.hk, generator=g)
        self.norm = torch.rand(self.hv, generator=g) + 0.5
        self.pitch = (self.hk * vdim + 3) // 4 * 4 + 4
        self.state = torch.zeros(6, self.pitch, device="cuda")
        self.seen = {}                      # slot -> lists of the recurrence's inputs (plain, float64)

    def open(self, slot):
        self.state[slot].zero_()
        self.seen[slot] = None

    def step(self, slots, lens, make=None, single=False):
        """One step; returns (engine rows [nt, H vdim], plain rows)."""
        lib, H, dim, vdim, rank, td, hk, hv = self.lib, self.H, self.dim, self.vdim, self.rank, self.td, self.hk, self.hv
        nt, eps, tau = sum(lens), 1e-5, 3.0
        # r | k | v | gate for the delta rule (vdim equals dim), q | k | v | gate for the gated linear attention
        parts = [torch.randn(nt, H, n, generator=self.g) for n in (dim, dim, vdim, vdim)]
        az = torch.randn(nt, hk + rank, generator=self.g)       # removal rate | the decay's first projection
        if make is not None:
            make(parts, az)
        parts = [p.to(td) for p in parts]
        z = torch.cat([p.reshape(nt, -1) for p in parts], 1).contiguous()
        starts = [0]
        for n in lens:
            starts.append(starts[-1] + n)
        d_z, d_az, d_w0, d_ba, d_norm, d_w2 = (t.cuda() for t in (z, az, self.w0, self.ba, self.norm, self.w2))
        d_start, d_slots = _ints(starts), _ints(slots)
        ldz, ldy = z.shape[1], hv + 8
        y = torch.full((nt, ldy), 3.0, dtype=td, device="cuda")
        gla = self.kind == "gla"
        small = az[:, hk:].double() if gla else torch.tanh(az[:, hk:].double())
        state = (lib.ptr(self.state), self.pitch)
        where = (lib.ptr(d_start), lib.ptr(d_slots), nt, len(slots), H)
        if single and gla:
            lib.call("tb_gated_linear_step_" + self.sfx, lib.ptr(d_z), ldz, lib.ptr(d_az[:, hk:]), hk + rank, lib.ptr(d_w2),
                     lib.ptr(d_w0), lib.ptr(d_norm), *state, lib.ptr(y), ldy, *where, dim, vdim, rank, 1 / tau, dim ** -0.5, eps)
        elif single:
            lib.call("tb_split_delta_step_" + self.sfx, lib.ptr(d_z), ldz, lib.ptr(d_az), hk + rank, lib.ptr(d_ba),
                     lib.ptr(d_w2), lib.ptr(d_w0), lib.ptr(d_norm), eps, *state, lib.ptr(y), ldy, *where, dim, rank)
        else:
            from transformer_b200.parts.gated_linear import split_weight, split_width
            wide = split_width(rank, td)
            th = torch.empty(nt, wide, dtype=td, device="cuda")
            lib.call(("tb_split_rows_" if gla else "tb_decay_tanh_") + self.sfx, lib.ptr(d_az[:, hk:]), hk + rank, lib.ptr(th),
                     nt, rank, wide)
            pre = (th.double().cpu() @ split_weight(self.w2, td).double().T).float().cuda()
            o = torch.empty(nt, hv, device="cuda")
            if gla:
                size = lib.gated_linear_record_size(dim, vdim)
                rec = torch.empty(H, nt, size, device="cuda")
                lib.call("tb_gated_linear_prep_" + self.sfx, lib.ptr(d_z), ldz, lib.ptr(pre), lib.ptr(d_w0), lib.ptr(rec), nt, H,
                         dim, vdim, size, 1 / tau, dim ** -0.5)
                lib.call("tb_decay_scan_rect", lib.ptr(rec), *state, lib.ptr(o), *where, dim, vdim)
            else:
                rec = torch.empty(H, nt, lib.split_delta_record_size(dim), device="cuda")
                lib.call("tb_split_delta_prep_" + self.sfx, lib.ptr(d_z), ldz, lib.ptr(d_az), hk + rank, lib.ptr(d_ba),
                         lib.ptr(pre), lib.ptr(d_w0), lib.ptr(rec), nt, H, dim)
                lib.call("tb_split_delta_scan", lib.ptr(rec), *state, lib.ptr(o), *where, dim)
            lib.call("tb_mlstm_out_" + self.sfx, lib.ptr(o), lib.ptr(d_z[:, ldz - hv:]), ldz, lib.ptr(d_norm), lib.ptr(y), nt, H,
                     vdim, eps, 1 if gla else 0, ldy)
        torch.cuda.synchronize()
        w = {"a1": torch.eye(rank, dtype=torch.float64), "w1": torch.eye(rank, dtype=torch.float64), "a2": self.w2.double(),
             "w2": self.w2.double(), "a2.b": self.w0.double(), "w0": self.w0.double()}
        pre_in = az[:, hk:].double()
        dec = (TP.gla_decay(pre_in, w, tau) if gla else TP.right_decay(pre_in, w)).view(nt, H, dim)
        a = torch.sigmoid(az[:, :hk].double() + self.ba.double()).view(nt, H, dim)
        f = [p.double() for p in parts]
        ins = [f[0] * dim ** -0.5, f[1], f[2], dec] if gla else [f[0], dec, f[1], f[2], a]
        want = torch.empty(nt, hv, dtype=torch.float64)
        for b, s in enumerate(slots):
            lo, hi = starts[b], starts[b + 1]
            new, old = [t[lo:hi] for t in ins], self.seen[s]
            self.seen[s] = new if old is None else [torch.cat([p, q]) for p, q in zip(old, new)]
            full = (TP.gla_recurrence if gla else TP.right_recurrence)(*self.seen[s])[-(hi - lo):]
            gate = f[3][lo:hi].reshape(hi - lo, hv)
            want[lo:hi] = TP.rms(full, eps).reshape(hi - lo, hv) * self.norm.double() * \
                (TP.silu(gate) if gla else torch.sigmoid(gate))
        assert bool((self.state[:, hk * vdim:] == 0).all()), "entries beside a slot's memory were written"
        got = y.cpu()
        assert bool((got[:, hv:] == 3.0).all()), "entries beside the heads' were written"
        return got[:, :hv].double(), want


SIZES = [("gla", 2, 64, 64, 16), ("gla", 1, 128, 48, 64), ("gla", 3, 7, 11, 5), ("gla", 2, 33, 30, 12), ("gla", 1, 256, 128, 8),
         ("gla", 4, 16, 256, 8), ("gla", 2, 48, 64, 24), ("gla", 24, 64, 64, 8), ("gla", 12, 128, 160, 8),
         ("delta", 2, 64, 64, 16), ("delta", 1, 128, 128, 64), ("delta", 3, 7, 7, 5), ("delta", 2, 33, 33, 12),
         ("delta", 1, 127, 127, 8), ("delta", 4, 16, 16, 8), ("delta", 2, 48, 48, 24), ("delta", 2, 96, 96, 8),
         ("delta", 24, 64, 64, 8), ("delta", 12, 128, 128, 8), ("delta", 2, 2, 2, 3)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind, H, dim, vdim, rank", SIZES + [("delta", 1, 256, 256, 8)])
def test_memory_carried_over_prompts_portions_and_single_tokens(dtype, kind, H, dim, vdim, rank):
    m = _Memory(kind, dtype, H, dim, vdim, rank, H + dim)
    tol = 1e-3 if dtype == "float32" else 4e-2
    for s in (3, 1, 5):
        m.open(s)
    one = dim <= 128 or kind == "gla"       # larger heads of the delta rule take the scan for single tokens too
    plan = [([3, 1, 5], [17, 1, 40], False), ([3, 1, 5], [1, 1, 1], one), ([5, 3], [8, 2], False), ([1], [1], one),
            ([1, 3], [23, 1], False), ([5, 1, 3], [1, 1, 1], one), ([3], [1], False)]
    for i, (slots, lens, single) in enumerate(plan):
        got, want = m.step(slots, lens, single=single)
        scale = max(1.0, float(want.abs().max()))
        assert float((got - want).abs().max()) <= tol * scale, f"step {i}: {float((got - want).abs().max()):.3e} of {scale:.2f}"
    m.open(3)                               # the slot again, for another sequence
    got, want = m.step([3], [9])
    assert float((got - want).abs().max()) <= tol * max(1.0, float(want.abs().max())), "a slot used again"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("single", [False, True])
@pytest.mark.parametrize("kind", ["gla", "delta"])
def test_memory_gives_back_what_was_written_long_ago(dtype, single, kind):
    """One strong write under key channel 5 whose decay is next to none, 300 tokens that write (and remove) elsewhere, then
    a question for that channel, in another step and in a used slot: the answer is the value that was written."""
    H, dim, rank = 2, 64, 8
    m = _Memory(kind, dtype, H, dim, dim, rank, 7)
    m.w2.zero_()
    m.w0 = torch.full((H * dim,), 1.0)
    m.w0.view(H, dim)[:, 5] = 14.0 if kind == "gla" else -14.0         # keeps
    m.open(2)
    m.step([2], [30])
    m.open(2)
    value = torch.randn(H, dim, generator=m.g)

    def write(p, az):
        p[1].zero_()
        p[1][0, :, 5], p[2][0] = 4.0, value

    def elsewhere(p, az):
        p[1][:, :, 5] = 0

    def ask(p, az):
        p[0].zero_(), p[1].zero_()
        p[0][:, :, 5], p[3][:] = 1.0, 2.0

    m.step([2], [1], write, single=single)
    m.step([2], [300], elsewhere)
    got, want = m.step([2], [1], ask, single=single)
    tol = 1e-3 if dtype == "float32" else 4e-2
    assert float((got - want).abs().max()) <= tol * float(want.abs().max())
    v = value.to(m.td).double()
    gate = TP.silu(torch.tensor(2.0, dtype=torch.float64)) if kind == "gla" else torch.sigmoid(torch.tensor(2.0, dtype=torch.float64))
    direct = TP.rms(v * 4.0, 0.0).reshape(-1) * m.norm.double() * gate
    assert float((got[0] - direct).abs().max()) <= 5e-2 * float(direct.abs().max())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("single", [False, True])
def test_a_key_written_twice_holds_the_second_value(dtype, single):
    """The removal takes away what lies under a key before the next value is written there: with a rate of one and next to
    no decay the second value is all that is left, with a rate of zero both are."""
    H, dim, rank = 2, 32, 4
    for rate, weight in ((30.0, 0.0), (-30.0, 1.0)):
        m = _Memory("delta", dtype, H, dim, dim, rank, 3)
        m.w2.zero_()
        m.w0, m.ba = torch.full((H * dim,), -30.0), torch.full((H * dim,), rate)
        m.open(0)
        key = torch.zeros(dim)
        key[3], key[9] = 2.0, -1.0
        values = [torch.randn(H, dim, generator=m.g) for _ in range(2)]

        def write(v, p, az):
            p[0][:], p[1][:], p[2][0], p[3][:] = key, key, v, 40.0
        m.step([0], [1], lambda p, az: write(values[0], p, az), single=single)
        got, want = m.step([0], [1], lambda p, az: write(values[1], p, az), single=single)
        tol = 1e-3 if dtype == "float32" else 4e-2
        assert float((got - want).abs().max()) <= tol * float(want.abs().max())
        left = [v.to(m.td).double() for v in values]
        direct = TP.rms((left[1] + weight * left[0]) * 5.0, 1e-5).reshape(-1) * m.norm.double()
        assert float((got[0] - direct).abs().max()) <= 5e-2 * float(direct.abs().max())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n, d", [(6, 48), (5, 50), (300, 192), (3, 4096), (2, 13001), (0, 64)])
def test_stream_step_in_all_its_forms(dtype, n, d):
    """The delta with and without its bias and its gate (whose rows have a pitch), with and without a sum over the depth,
    with the norm, without it and without an output, for all rows and for chosen ones."""
    from transformer_b200.csrc import lib
    td, sfx = _td(dtype)
    g = torch.Generator().manual_seed(d)
    pad = 8
    x0, delta = torch.randn(n, d, generator=g) * 2, (torch.randn(n, d, generator=g) * 3).to(td)
    gate, gb, db = (torch.randn(n, d + pad, generator=g) * 2).to(td), torch.randn(d, generator=g), torch.randn(d, generator=g)
    hist0, c = torch.randn(5, n, d, generator=g), torch.randn(5, generator=g)
    alpha, w, b = torch.tensor([0.7]), torch.randn(d, generator=g), torch.randn(d, generator=g)
    chosen = [n - 1, 0] if n else []
    d_delta, d_gate, d_gb, d_db, d_c, d_alpha, d_w, d_b = (t.cuda() for t in (delta, gate, gb, db, c, alpha, w, b))
    d_rows = _ints(chosen)
    for has_delta, has_db, has_gate, has_gb in ((0, 0, 0, 0), (1, 0, 0, 0), (1, 1, 0, 0), (1, 0, 1, 1), (1, 1, 1, 1), (1, 1, 1, 0)):
        for terms in (0, 1, 2, 5):
            for out in ("norm", "rows", "stream", "nothing"):
                x, hist = x0.clone().cuda(), hist0.clone().cuda()
                rows = chosen if out == "rows" else list(range(n))
                y = torch.full((len(rows), d), 5.0, dtype=td, device="cuda")
                norm = out in ("norm", "rows")
                lib.call("tb_stream_step_" + sfx, lib.ptr(x), lib.ptr(d_delta) if has_delta else 0, lib.ptr(d_db) if has_db else 0,
                         lib.ptr(d_gate) if has_gate else 0, d + pad if has_gate else 0, lib.ptr(d_gb) if has_gb else 0,
                         lib.ptr(hist) if terms else 0, hist.stride(0) if terms else 0, lib.ptr(d_c) if terms else 0, terms,
                         lib.ptr(d_rows) if out == "rows" else 0, lib.ptr(d_alpha) if norm else 0, lib.ptr(d_w) if norm else 0,
                         lib.ptr(d_b) if norm else 0, 0 if out == "nothing" else lib.ptr(y), len(rows), d)
                torch.cuda.synchronize()
                if not n:
                    continue
                v = x0.double()
                if has_delta:
                    u = delta.double() + (db.double() if has_db else 0)
                    if has_gate:
                        u = u * torch.sigmoid(gate[:, :d].double() + (gb.double() if has_gb else 0))
                    v = v + u
                want_hist = hist0.double().clone()
                if terms:
                    h = want_hist.clone()
                    h[terms - 1] = v
                    if out != "rows":
                        want_hist = h
                    v = torch.einsum("j,jnd->nd", c[:terms].double(), h[:terms])
                assert float((hist.cpu().double() - want_hist).abs().max()) < 1e-4
                want_x = x0.double() if out == "rows" else v
                assert float((x.cpu().double() - want_x).abs().max()) < 1e-4
                if out == "nothing":
                    assert bool((y == 5.0).all())
                    continue
                want = v[rows]
                if norm:
                    want = torch.tanh(0.7 * want) * w.double() + b.double()
                tol = 1e-4 if dtype == "float32" else 2.0 ** -8 * float(want.abs().max())
                assert float((y.cpu().double() - want).abs().max()) < tol, (has_gate, terms, out)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d", [48, 50, 2056])
def test_embedding_with_positions(dtype, d):
    from transformer_b200.csrc import lib
    td, sfx = _td(dtype)
    g = torch.Generator().manual_seed(d)
    table, pos = torch.randn(9, d, generator=g).to(td), torch.randn(20, d, generator=g).to(td)
    alpha, w, b = torch.tensor([0.6]), torch.randn(d, generator=g), torch.randn(d, generator=g)
    tok, at = [3, 0, 8, 3], [0, 19, 7, 1]
    dv = [t.cuda() for t in (table, pos, alpha, w, b)]
    d_tok, d_at = _ints(tok), _ints(at)
    for norm in (True, False):
        x = torch.empty(4, d, device="cuda")
        lib.call("tb_embed_learned_" + sfx, lib.ptr(d_tok), lib.ptr(d_at), lib.ptr(dv[0]), lib.ptr(dv[1]), lib.ptr(x), 4, d, 1.5,
                 *((lib.ptr(t) for t in dv[2:]) if norm else (0, 0, 0)))
        torch.cuda.synchronize()
        want = table.double()[tok] * 1.5 + pos.double()[at]
        if norm:
            want = torch.tanh(alpha.double() * want) * w.double() + b.double()
        assert float((x.cpu().double() - want).abs().max()) < 1e-5
