"""The Fofapel design in the engine against the plain implementation: each mechanism alone, prompts against decoding,
portions, unequal batches, reused slots and pages, the first tokens, windows' edges, long decoding, generation; and its
kernels alone with inputs made so that a fault shows."""
import json
import subprocess
import sys

import pytest
import torch

import fofapel_tiny as T
from plain import fofapel_plain as FP
from tiny import ROOT, TraceRun, random_prompts

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    tmp = tmp_path_factory.mktemp("fofapel")
    return {name: T.make_folder(tmp, name) for name in T.CONFIGS}


def _load(folder, dtype, **kw):
    import transformer_b200 as tb
    kw.setdefault("max_tokens", 2048)
    return tb.load(folder, dtype=dtype, **kw)


def _tokens(folder, n, seed):
    cfg, _ = FP.read_folder(folder)
    return random_prompts(cfg["vocab"], [n], seed)[0]


def greedy(cfg, tensors, prompt, steps):
    seq, out = list(prompt), []
    for _ in range(steps):
        tok = int(torch.argmax(FP.forward(cfg, tensors, seq)[-1]))
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
@pytest.mark.parametrize("name", ["left", "right", "dense", "experts", "shared"])
def test_each_mechanism_alone(name, dtype, folders):
    """One kind of part: every position of a prompt that crosses a page border, then six tokens decoded."""
    cfg, tensors = FP.read_folder(folders[name])
    tokens = _tokens(folders[name], 106, 11)
    rows = T.run_cuts(_load(folders[name], dtype), tokens, [100])
    T.check_request(cfg, tensors, tokens, rows, dtype, name)


@pytest.mark.parametrize("dtype", DTYPES)
def test_prompt_against_decoding_token_by_token(dtype, folders):
    cfg, tensors = FP.read_folder(folders["mixed"])
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
    """A prompt fed in portions, down to two tokens, with cuts at and beside page and window borders: the memory and the
    last input come from the step before, the window reaches back over several portions."""
    cfg, tensors = FP.read_folder(folders["mixed"])
    tokens = _tokens(folders["mixed"], 140, 6)
    rows = T.run_cuts(_load(folders["mixed"], dtype), tokens, cuts)
    T.check_request(cfg, tensors, tokens, rows, dtype, f"cuts {cuts}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_step_cut_into_pieces_by_the_engine(dtype, folders):
    cfg, tensors = FP.read_folder(folders["mixed"])
    tokens = _tokens(folders["mixed"], 100, 16)
    rows = T.run_cuts(_load(folders["mixed"], dtype, max_step_tokens=37), tokens, [95])
    T.check_request(cfg, tensors, tokens, rows, dtype, "pieces")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_unequal_batch_equals_each_request_alone(name, dtype, folders):
    """Prompts of 1, 63, 64 and 130 tokens in one step, then decoded together while the short ones end; in slots
    and pages that an earlier batch has used."""
    cfg, tensors = FP.read_folder(folders[name])
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
    """Sequences of one, two and three tokens side by side: the softmax of the first token holds one key and the sink,
    the shift reaches before the start, the memory is empty.  (The first token's heads are its values times the bonus,
    divided by their own size: the tokens are such that no bonus is close to zero.)"""
    cfg, tensors = FP.read_folder(folders["mixed"])
    engine = _load(folders["mixed"], dtype)
    seqs = [_tokens(folders["mixed"], n, 80 + n) for n in (1, 2, 3)]
    slots = [engine.open() for _ in seqs]
    lg = engine.step(slots, seqs, [list(range(len(s))) for s in seqs]).cpu()
    T.check_requests(cfg, tensors, [(seqs[0], {0: lg[0]}), (seqs[1], {0: lg[1], 1: lg[2]}),
                                    (seqs[2], {0: lg[3], 1: lg[4], 2: lg[5]})], dtype, "sequences of one to three")


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_through_graphs(dtype, folders):
    """Three prompt tokens, then 200 tokens decoded through the replayed step: every window fills and moves on, the
    memory is carried 200 times."""
    cfg, tensors = FP.read_folder(folders["mixed"])
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
    cfg, tensors = FP.read_folder(folders["wide"])
    T.check_requests(cfg, tensors, list(zip(seqs, got)), dtype, "20 sequences")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name, n, cuts", [("wide", 420, [410]), ("wide", 300, [70, 200]), ("odd", 90, [66, 3])])
def test_sizes_that_reach_the_fast_kernels_and_sizes_that_none_takes(name, n, cuts, dtype, folders):
    cfg, tensors = FP.read_folder(folders[name])
    tokens = _tokens(folders[name], n, 3)
    rows = T.run_cuts(_load(folders[name], dtype), tokens, cuts)
    T.check_request(cfg, tensors, tokens, rows, dtype, name)


@pytest.mark.parametrize("seed", [0, 1, 2, 3, 4, 5])
def test_configurations_drawn_at_random(seed, tmp_path):
    """Layers and sizes drawn at random (two of three draws take sizes that reach the vector and tensor-core forms): a
    prompt across several pages and twelve decoded tokens."""
    import random
    rng = random.Random(2000 + seed)
    cfg = T.random_config(rng, nice=seed % 3 != 2)
    folder = T.make_folder(tmp_path, f"drawn{seed}", cfg=cfg, seed=seed)
    cfg, tensors = FP.read_folder(folder)
    n = rng.randrange(150, 280)
    tokens = random_prompts(cfg["vocab"], [n + 12], seed)[0]
    for dtype in DTYPES:
        rows = T.run_cuts(_load(folder, dtype), tokens, [n])
        T.check_request(cfg, tensors, tokens, rows, dtype, f"drawn {seed}")


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


def test_a_table_that_names_an_expert_too_many_is_refused(tmp_path):
    def edit(t):
        t["l0.mlp.table"][3, 0] = 6
    folder = T.make_folder(tmp_path, "shared", tensors_edit=edit)
    with pytest.raises(ValueError, match="expert"):
        _load(folder, "float32")


def test_greedy_generation_through_the_entry_point(folders):
    import transformer_b200 as tb
    cfg, tensors = FP.read_folder(folders["mixed"])
    prompts = [_tokens(folders["mixed"], n, 30 + n) for n in (7, 66, 2)]
    got = tb.generate(_load(folders["mixed"], "float32"), prompts, max_steps=6, stop_tokens=()).tokens
    assert got == [greedy(cfg, tensors, p, 6) for p in prompts]
    res = tb.generate(_load(folders["mixed"], "bfloat16"), prompts, max_steps=6, stop_tokens=())
    assert [len(t) for t in res.tokens] == [6, 6, 6]


def test_trace_runner_and_command_line(folders, tmp_path):
    cfg, tensors = FP.read_folder(folders["mixed"])
    a, b = _tokens(folders["mixed"], 70, 1), _tokens(folders["mixed"], 9, 2)
    run = TraceRun(folders["mixed"], "float32", str(tmp_path / "out"), 256, record_routing=False)
    run.step(0, [{"id": "a", "tokens": a[:66], "want": [0, 65]}, {"id": "b", "tokens": b[:8], "want": [7]}])
    run.step(1, [{"id": "a", "tokens": a[66:67], "want": [0]}, {"id": "b", "tokens": b[8:9], "want": []}], end=["b"])
    run.step(2, [{"id": "a", "tokens": a[67:68], "want": [0]}], end=["a"])
    first, second, third = (run.logits(i, cfg["vocab"]) for i in range(3))
    run.close()
    ref_a, ref_b = FP.forward(cfg, tensors, a), FP.forward(cfg, tensors, b)
    for got, want in ((first[0], ref_a[0]), (first[1], ref_a[65]), (first[2], ref_b[7]), (second[0], ref_a[66]),
                      (third[0], ref_a[67])):
        assert float((got.double() - want).abs().max()) <= T.FP32_TOL
    assert second.shape[0] == 1
    out = subprocess.run([sys.executable, "-m", "transformer_b200", "generate", "--model", folders["mixed"],
                          "--prompt", " ".join(map(str, b)), "--max-steps", "4", "--dtype", "float32", "--json"],
                         cwd=ROOT, capture_output=True, text=True, timeout=600)
    assert out.returncode == 0, out.stderr[-2000:]
    assert json.loads(out.stdout.strip().splitlines()[-1])["tokens"] == [greedy(cfg, tensors, b, 4)]


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


def _edge(which, p, window, g):
    j = {"oldest inside": p - window + 1, "newest outside": p - window, "page row 63": p // 64 * 64 - 1,
         "page row 64": p // 64 * 64, "itself": p, "far": p - 300}[which]
    return min(max(j, 0), p)


@pytest.mark.parametrize("kernel, dtype, splits", [("general", "float32", 1), ("general", "float32", 3), ("general", "bfloat16", 1),
                                                   ("mma", "bfloat16", 1), ("mma", "bfloat16", 3)])
@pytest.mark.parametrize("H, G, dim, window", [(4, 2, 64, 96), (6, 2, 32, 64), (2, 2, 128, 65), (8, 1, 64, 1), (3, 1, 96, 1 << 30)])
def test_windowed_attention_with_head_gates_and_a_pitch(kernel, dtype, splits, H, G, dim, window):
    """Every head asks, far above the rest, for one key (the oldest inside its window, the newest outside, a page's last
    or first row, itself, one 300 tokens back), with a sink of score zero, one gate per head, a multiplier, and rows that
    are a part of wider ones whose other entries stay as they were."""
    from transformer_b200.csrc import lib
    td, sfx = _td(dtype)
    g = torch.Generator().manual_seed(H * dim + splits)
    pg = _Pages([0, 130, 64, 321, 40], [90, 1, 1, 1, 70], g)
    kc = torch.randn(pg.n_pages, G, 64, dim, generator=g).to(td)
    vc = torch.randn(pg.n_pages, G, 64, dim, generator=g).to(td)
    keys, vals = [], []
    for b, n in enumerate(pg.total):
        k = torch.randn(n, G, dim, generator=g)
        k, v = (k / k.norm(dim=-1, keepdim=True)).to(td), torch.randn(n, G, dim, generator=g).to(td)
        pg.put(kc, b, 0, k)
        pg.put(vc, b, 0, v)
        keys.append(k.double())
        vals.append(v.double())
    gz = (torch.randn(pg.nt, H + 5, generator=g) * 2).to(td)
    d_kc, d_vc, d_gz, sinks = kc.cuda(), vc.cuda(), gz.cuda(), torch.zeros(H, device="cuda")
    ldo, scale, mult = H * dim + 8, 0.5, 1.25
    tq = lib.attention_window_mma_tile_tokens(H, G) if kernel == "mma" else lib.attention_tile_tokens(H, G)
    t_seq, t_t0, t_nq, count = pg.tiles(tq)
    for which in ("oldest inside", "newest outside", "page row 63", "page row 64", "itself", "far", "any"):
        q, want = torch.zeros(pg.nt, H, dim), torch.zeros(pg.nt, H, dim, dtype=torch.float64)
        for b in range(len(pg.new)):
            for i in range(pg.new[b]):
                p, t = pg.before[b] + i, pg.starts[b] + i
                for h in range(H):
                    q[t, h] = torch.randn(dim, generator=g) * 4 if which == "any" else \
                        keys[b][_edge(which, p, min(window, 1000), g), h // (H // G)].float() * 24.0
                    qh = q[t, h].to(td).double()
                    lo = max(0, p - window + 1)
                    w = FP.softmax_off_by_one(keys[b][lo:p + 1, h // (H // G)] @ qh * scale)
                    want[t, h] = w @ vals[b][lo:p + 1, h // (H // G)] * torch.sigmoid(gz[t, 5 + h].double()) * mult
        d_q = q.to(td).cuda()
        out = torch.full((pg.nt, ldo), 7.0, dtype=td, device="cuda")
        partial = torch.empty(pg.nt, H, splits, dim + 2, device="cuda")
        name = "tb_attention_window_mma_heads_bf16" if kernel == "mma" else "tb_attention_window_heads_" + sfx
        ok = lib.try_call(name, lib.ptr(d_q), lib.ptr(out), lib.ptr(d_kc), lib.ptr(d_vc), lib.ptr(d_gz[:, 5:]),
                          lib.ptr(t_seq), lib.ptr(t_t0), lib.ptr(t_nq), lib.ptr(pg.tok_pos), lib.ptr(pg.table),
                          lib.ptr(partial) if splits > 1 else 0, count, pg.nt, pg.max_pages, H * dim, H + 5, H, G, dim, dim,
                          splits, window, 0, scale, 0.0, 0, lib.ptr(sinks), 0, 0, 1, mult, ldo)
        assert ok, "the kernel refused sizes it is meant to take"
        torch.cuda.synchronize()
        got = out.cpu()
        assert bool((got[:, H * dim:] == 7.0).all()), "entries beside the heads' were written"
        diff = (got[:, :H * dim].double().view(pg.nt, H, dim) - want).abs()
        assert float(diff.max()) <= (2e-5 if dtype == "float32" else 4e-2), f"{which}: {float(diff.max()):.3e}"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H, G, dim, rdims, lens", [(4, 2, 64, 64, [70, 3]), (3, 1, 10, 6, [5, 66]), (6, 3, 24, 0, [1, 1]),
                                                    (2, 2, 256, 128, [80, 1]), (5, 5, 7, 4, [40, 30])])
def test_head_kernel_for_values_that_are_the_keys(dtype, H, G, dim, rdims, lens):
    """Biases, rotation, the norm without weights and the cache write: queries and keys normed, values the biased key as
    it is, every row in its page and nowhere else."""
    from transformer_b200.csrc import lib
    from transformer_b200.parts.rope import Rope
    td, sfx = _td(dtype)
    g = torch.Generator().manual_seed(dim + H)
    pg = _Pages([62, 130], lens, g)
    ldz = (H + G) * dim + H + 1
    z = torch.randn(pg.nt, ldz, generator=g).to(td)
    bias = torch.randn((H + G) * dim, generator=g)
    kc = torch.full((pg.n_pages, G, 64, dim), 9.0, dtype=td, device="cuda")
    vc = kc.clone()
    qo = torch.empty(pg.nt, H * dim, dtype=td, device="cuda")
    cos = sin = None
    if rdims:
        cos, sin = Rope({"dh": rdims, "theta": 100.0, "positions": 256}, td, torch.device("cuda")).tables()
    d_z, d_b = z.cuda(), bias.cuda()
    lib.call("tb_head_prep_keyed_" + sfx, lib.ptr(d_z), ldz, lib.ptr(d_b), 1, 1e-3, lib.ptr(cos), lib.ptr(sin), lib.ptr(qo),
             lib.ptr(kc), lib.ptr(vc), lib.ptr(pg.tok_seq), lib.ptr(pg.tok_pos), lib.ptr(pg.seq_start), lib.ptr(pg.table),
             pg.max_pages, pg.nt, H, G, dim, rdims)
    torch.cuda.synchronize()
    u = (z[:, :(H + G) * dim].double() + bias.double()).view(pg.nt, H + G, dim)
    want_k, want_v = torch.full(kc.shape, 9.0, dtype=torch.float64), torch.full(kc.shape, 9.0, dtype=torch.float64)
    tol = 1e-5 if dtype == "float32" else 2e-2
    for b, n in enumerate(pg.new):
        for i in range(n):
            t, p = pg.starts[b] + i, pg.before[b] + i
            y = FP.rms(FP.rotate_pairs(u[t], p, rdims, 100.0), 1e-3)
            assert float((qo[t].cpu().double().view(H, dim) - y[:H]).abs().max()) <= tol, f"query of token {t}"
            pg.put(want_k, b, p, [y[H:]])
            pg.put(want_v, b, p, [u[t, H:]])
    assert float((kc.cpu().double() - want_k).abs().max()) <= tol
    assert float((vc.cpu().double() - want_v).abs().max()) <= tol * 3
