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


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d", [40, 50, 1032])
def test_mixes_with_the_token_before(dtype, d):
    """All five mixes; a portion's first token reads the slot's last input, whichever tile it falls into; the lists by
    which a grouped product takes the first four."""
    from transformer_b200.csrc import lib
    td, sfx = _td(dtype)
    g = torch.Generator().manual_seed(d)
    mu = torch.rand(5, d, generator=g)
    size = lib.decay_state_size(2, 6, d)
    state = torch.randn(7, size, generator=g)
    d_mu, d_state = mu.cuda(), state.cuda()
    for lens in ([1, 1, 1], [3, 1, 5], [130, 7, 190]):
        nt = sum(lens)
        slots = [4, 0, 6]
        x = torch.randn(nt, d, generator=g).to(td)
        pg = _Pages([0] * 3, lens, g)
        out = torch.empty(5, nt, d, dtype=td, device="cuda")
        offsets, groups = _ints([0] * 5), _ints([9] * (4 * nt))
        d_x, d_slots = x.cuda(), _ints(slots)
        lib.call("tb_shift_mix_" + sfx, lib.ptr(d_x), lib.ptr(d_mu), lib.ptr(d_state), size, 2 * 6 * 6, lib.ptr(out),
                 lib.ptr(offsets), lib.ptr(groups), 4, lib.ptr(pg.tok_seq), lib.ptr(pg.seq_start), lib.ptr(d_slots), nt, d)
        torch.cuda.synchronize()
        before = torch.cat([torch.cat([state[s, 72:72 + d][None].double(), x[a:b - 1].double()])
                            for s, a, b in zip(slots, pg.starts, pg.starts[1:])])
        want = x.double()[None] + (before - x.double())[None] * mu.double()[:, None]
        assert float((out.cpu().double() - want).abs().max()) <= (1e-5 if dtype == "float32" else 3e-2)
        assert offsets.cpu().tolist() == [j * nt for j in range(5)]
        assert groups.cpu().tolist() == [j for j in range(4) for _ in range(nt)]


class _Memory:
    """The recurrence's kernels over a batch in slots, carried from step to step, beside the plain recurrence."""

    def __init__(self, dtype, H, dim, rank, width, seed):
        from transformer_b200.csrc import lib
        self.lib, (self.td, self.sfx) = lib, _td(dtype)
        self.H, self.dim, self.rank, self.width = H, dim, rank, width
        g = self.g = torch.Generator().manual_seed(seed)
        hd = H * dim
        self.w2 = (torch.randn(hd, rank, generator=g) * rank ** -0.5).to(self.td)
        self.w0, self.u = torch.rand(hd, generator=g) * 4 - 4, torch.randn(H, dim, generator=g)
        self.norm = torch.rand(hd, generator=g) + 0.5
        size = lib.decay_state_size(H, dim, width)
        self.pitch = size
        self.state = torch.zeros(6, size, device="cuda")
        self.seen = {}                      # slot -> lists of r, k, v, dec (plain, float64)

    def open(self, slot):
        self.state[slot].zero_()
        self.seen[slot] = None

    def step(self, slots, lens, make=None, single=False):
        """One step; returns (engine rows [nt, H, dim] before the gate's effect is taken off, plain rows)."""
        lib, H, dim, rank, td = self.lib, self.H, self.dim, self.rank, self.td
        nt, hd = sum(lens), H * dim
        z = torch.randn(4, nt, hd, generator=self.g)
        a = torch.randn(nt, rank, generator=self.g)
        if make is not None:
            make(z.view(4, nt, H, dim), a)
        z = z.to(td)
        x = torch.randn(nt, self.width, generator=self.g).to(td)
        starts = [0]
        for n in lens:
            starts.append(starts[-1] + n)
        dev = lambda t: t.cuda()
        d_z, d_a, d_x, d_w0, d_u, d_norm = map(dev, (z, a, x, self.w0, self.u, self.norm))
        d_start, d_slots = _ints(starts), _ints(slots)
        ldy = hd + 8
        y = torch.full((nt, ldy), 3.0, dtype=td, device="cuda")
        if single:
            d_w2 = self.w2.cuda()
            lib.call("tb_decay_step_" + self.sfx, lib.ptr(d_z), lib.ptr(d_x), self.width, lib.ptr(d_a), rank, lib.ptr(d_w2),
                     lib.ptr(d_w0), lib.ptr(d_u), lib.ptr(d_norm), 1e-5, lib.ptr(self.state), self.pitch, lib.ptr(y), ldy,
                     lib.ptr(d_start), lib.ptr(d_slots), nt, len(slots), H, dim, rank)
        else:
            half = (rank + 3) // 4 * 4
            wide = rank if td == torch.float32 else 2 * half
            th = torch.empty(nt, wide, dtype=td, device="cuda")
            lib.call("tb_decay_tanh_" + self.sfx, lib.ptr(d_a), rank, lib.ptr(th), nt, rank, wide)
            t64 = th.double().cpu()
            got_tanh = t64[:, :rank] if td == torch.float32 else t64[:, :rank] + t64[:, half:half + rank]
            assert float((got_tanh - torch.tanh(a.double())).abs().max()) <= (1e-6 if td == torch.float32 else 1e-5)
            pre = (got_tanh @ self.w2.double().T).float().cuda()
            rec = torch.empty(H, nt, lib.decay_record_size(dim), device="cuda")
            o = torch.empty(nt, hd, device="cuda")
            lib.call("tb_decay_prep_" + self.sfx, lib.ptr(d_z), lib.ptr(pre), lib.ptr(d_w0), lib.ptr(d_u), lib.ptr(rec),
                     nt, H, dim)
            lib.call("tb_decay_scan_" + self.sfx, lib.ptr(rec), lib.ptr(self.state), self.pitch, lib.ptr(o),
                     lib.ptr(d_x), self.width, lib.ptr(d_start), lib.ptr(d_slots), nt, len(slots), H, dim)
            lib.call("tb_mlstm_out_" + self.sfx, lib.ptr(o), lib.ptr(d_z[3]), hd, lib.ptr(d_norm), lib.ptr(y), nt, H, dim,
                     1e-5, 1, ldy)
        torch.cuda.synchronize()
        dec = torch.exp(-torch.exp(torch.tanh(a.double()) @ self.w2.double().T + self.w0.double()))
        want = torch.empty(nt, hd, dtype=torch.float64)
        for b, s in enumerate(slots):
            lo, hi = starts[b], starts[b + 1]
            new = [t[lo:hi].double().view(hi - lo, H, dim) for t in (z[0], z[1], z[2], dec)]
            old = self.seen[s]
            self.seen[s] = new if old is None else [torch.cat([p, q]) for p, q in zip(old, new)]
            full = FP.recurrence(*self.seen[s], self.u.double())[-(hi - lo):]
            want[lo:hi] = FP.rms(full, 1e-5).reshape(hi - lo, hd) * self.norm.double() * FP.silu(z[3, lo:hi].double())
            last = self.state[s, H * dim * dim:H * dim * dim + self.width].cpu()
            assert torch.equal(last, x[hi - 1].float()), "the slot's last input"
        got = y.cpu()
        assert bool((got[:, hd:] == 3.0).all()), "entries beside the heads' were written"
        return got[:, :hd].double(), want


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H, dim, rank", [(2, 64, 16), (1, 128, 64), (3, 7, 5), (2, 33, 12), (1, 256, 8), (4, 16, 8), (2, 96, 24), (24, 64, 8), (12, 128, 8)])
def test_memory_carried_over_prompts_portions_and_single_tokens(dtype, H, dim, rank):
    m = _Memory(dtype, H, dim, rank, 50, H + dim)
    tol = 1e-3 if dtype == "float32" else 4e-2
    for s in (3, 1, 5):
        m.open(s)
    plan = [([3, 1, 5], [17, 1, 40], False), ([3, 1, 5], [1, 1, 1], True), ([5, 3], [8, 2], False), ([1], [1], True),
            ([1, 3], [23, 1], False), ([5, 1, 3], [1, 1, 1], True), ([3], [1], False)]
    for i, (slots, lens, single) in enumerate(plan):
        got, want = m.step(slots, lens, single=single)
        scale = max(1.0, float(want.abs().max()))
        assert float((got - want).abs().max()) <= tol * scale, f"step {i}: {float((got - want).abs().max()):.3e} of {scale:.2f}"
    m.open(3)                               # the slot again, for another sequence
    got, want = m.step([3], [9])
    assert float((got - want).abs().max()) <= tol * max(1.0, float(want.abs().max())), "a slot used again"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("single", [False, True])
def test_memory_gives_back_what_was_written_long_ago(dtype, single):
    """One strong write under key channel 5 whose decay is next to none, 300 tokens that write elsewhere, then a question
    for that channel, in another step and in a used slot: the answer is the value that was written, whatever the gates."""
    H, dim, rank = 2, 64, 8
    m = _Memory(dtype, H, dim, rank, 40, 7)
    m.w2.zero_()
    m.w0 = torch.full((H * dim,), -1.0)
    m.w0.view(H, dim)[:, 5] = -12.0         # keeps
    m.open(2)
    m.step([2], [30])
    m.open(2)
    value = torch.randn(H, dim, generator=m.g)

    def write(z, a):
        z[1] = 0
        z[1, 0, :, 5], z[2, 0] = 4.0, value

    def elsewhere(z, a):
        z[1, :, :, 5] = 0

    def ask(z, a):
        z[0] = 0
        z[0, :, :, 5], z[1], z[3] = 1.0, 0, 2.0

    m.step([2], [1], write, single=single)
    m.step([2], [300], elsewhere)
    got, want = m.step([2], [1], ask, single=single)
    tol = 1e-3 if dtype == "float32" else 4e-2
    assert float((got - want).abs().max()) <= tol * float(want.abs().max())
    v = value.to(m.td).double()
    direct = FP.rms(v * 4.0, 0.0).reshape(-1) * m.norm.double() * FP.silu(torch.tensor(2.0, dtype=torch.float64))
    assert float((got[0] - direct).abs().max()) <= 5e-2 * float(direct.abs().max())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d", [48, 50, 192, 4096, 6008, 13000])
def test_stream_norm_in_all_its_forms(dtype, d):
    """x <- y = N(alpha x + u): the delta a tensor or experts' rows; with and without what rides along (the table's
    experts, equal weights, the shared expert's gate from the row as stored)."""
    from transformer_b200.csrc import lib
    td, sfx = _td(dtype)
    g = torch.Generator().manual_seed(d)
    n, k, terms, vocab = 6, 3, 4, 11
    x0, delta = torch.randn(n, d, generator=g) * 2 + 0.5, (torch.randn(n, d, generator=g) * 3 + 1).to(td)
    w, b = torch.rand(d, generator=g) + 0.5, torch.randn(d, generator=g)
    ey, tw = torch.randn(n * terms, d, generator=g).to(td), torch.rand(n, terms, generator=g)
    at = torch.randperm(n * terms, generator=g).to(torch.int32)
    tok = torch.randint(0, vocab, (n,), generator=g).to(torch.int32)
    table = torch.randint(0, 99, (vocab, k), generator=g).to(torch.int32)
    gw = (torch.randn(d, generator=g) * d ** -0.5).to(td)
    dv = [t.cuda() for t in (delta, w, b, ey, tw, at, tok, table, gw)]
    d_delta, d_w, d_b, d_ey, d_tw, d_at, d_tok, d_table, d_gw = dv
    for rows in (False, True):
        for ride in ("nothing", "table", "table and gate"):
            x, y = x0.clone().cuda(), torch.empty(n, d, dtype=td, device="cuda")
            kk = k + (ride == "table and gate")
            idx, wts = torch.full((n, k), -1, dtype=torch.int32, device="cuda"), torch.full((n, kk), -1.0, device="cuda")
            pick = (0, 0, 0, 0, 0, 0) if ride == "nothing" else \
                (lib.ptr(d_tok), lib.ptr(d_table), lib.ptr(d_gw) if kk > k else 0, lib.ptr(idx), lib.ptr(wts), k)
            lib.call("tb_renew_layernorm_" + sfx, lib.ptr(x), 0 if rows else lib.ptr(d_delta), lib.ptr(d_ey) if rows else 0,
                     lib.ptr(d_at) if rows else 0, lib.ptr(d_tw) if rows else 0, terms if rows else 0, 1.75, lib.ptr(d_w),
                     lib.ptr(d_b), 1e-5, lib.ptr(y), n, d, *pick)
            torch.cuda.synchronize()
            u = torch.stack([sum(tw[t, j].double() * ey[at[t * terms + j]].double() for j in range(terms)) for t in range(n)]) \
                if rows else delta.double()
            want = FP.layer_norm(1.75 * x0.double() + u, w.double(), b.double(), 1e-5)
            assert float((x.cpu().double() - want).abs().max()) < 3e-5, "the stream itself is float"
            assert torch.equal(y.cpu(), x.cpu().to(td)), "the rows are the stream, rounded once"
            if ride == "nothing":
                continue
            assert torch.equal(idx.cpu(), table[tok.long()])
            assert float((wts[:, :k].cpu() - 1.0 / k).abs().max()) < 1e-7
            if kk > k:
                gate = torch.sigmoid(y.cpu().double() @ gw.double())
                assert float((wts[:, k].cpu().double() - gate).abs().max()) < 1e-5


@pytest.mark.parametrize("dtype", DTYPES)
def test_terms_and_lists_of_experts_with_a_shared_one(dtype):
    from transformer_b200.csrc import lib
    td, sfx = _td(dtype)
    g = torch.Generator().manual_seed(1)
    for nt, k, E, d in ((1, 1, 3, 40), (700, 2, 5, 50), (40, 4, 4, 128)):
        x, gw = torch.randn(nt, d, generator=g).to(td), (torch.randn(d, generator=g) * d ** -0.5).to(td)
        tok = torch.randint(0, 9, (nt,), generator=g).to(torch.int32)
        table = torch.stack([torch.randperm(E, generator=g)[:k] for _ in range(9)]).to(torch.int32)
        w_in = torch.rand(nt, k, generator=g)
        d_x, d_gw, d_tok, d_table, d_win = x.cuda(), gw.cuda(), tok.cuda(), table.cuda(), w_in.cuda()
        idx, wts = torch.zeros(nt, k, dtype=torch.int32, device="cuda"), torch.zeros(nt, k + 1, device="cuda")
        lib.call("tb_moe_terms_" + sfx, lib.ptr(d_x), lib.ptr(d_gw), lib.ptr(d_tok), lib.ptr(d_table), 0, lib.ptr(idx),
                 lib.ptr(wts), nt, d, k)
        gate = torch.sigmoid(x.double() @ gw.double())
        assert torch.equal(idx.cpu(), table[tok.long()]) and float((wts[:, :k].cpu() - 1 / k).abs().max()) < 1e-7
        assert float((wts[:, k].cpu().double() - gate).abs().max()) < 1e-5
        lib.call("tb_moe_terms_" + sfx, lib.ptr(d_x), 0, 0, 0, lib.ptr(d_win), 0, lib.ptr(wts), nt, d, k)
        assert torch.equal(wts.view(-1)[:nt * k].cpu(), w_in.view(-1))
        M = nt * k
        off, st, at = _ints([0] * (E + 1)), _ints([0] * M), _ints([-1] * (nt * (k + 1)))
        lib.call("tb_moe_dispatch_shared", lib.ptr(idx), lib.ptr(off), lib.ptr(st), lib.ptr(at), M, k, E)
        off, st, at, ex = off.cpu(), st.cpu(), at.cpu().view(nt, k + 1), idx.cpu()
        assert at[:, k].tolist() == [M + t for t in range(nt)] and sorted(at[:, :k].reshape(-1).tolist()) == list(range(M))
        for t in range(nt):
            for j in range(k):
                r, e = int(at[t, j]), int(ex[t, j])
                assert int(off[e]) <= r < int(off[e + 1]) and int(st[r]) == t


def test_tanh_gelu_pair_in_every_product():
    from transformer_b200.parts.linear import GELU_TANH, gemm_simt, gemm_skinny, gemm_tc
    g = torch.Generator().manual_seed(0)
    for M, K, N in ((5, 64, 40), (300, 128, 96)):
        a, w = torch.randn(M, K, generator=g) * 3, torch.randn(2 * N, K, generator=g) * K ** -0.5

        def want(a, w):
            p = a.double() @ w.double().T
            return FP.gelu_tanh(p[:, :N]) * p[:, N:]

        out = torch.empty(M, N, device="cuda")
        d_a, d_w = a.cuda(), w.cuda()
        gemm_simt(d_a, d_w, out, out_kind=2, glu=GELU_TANH)
        ref = want(a, w)
        assert float((out.cpu().double() - ref).abs().max()) <= 2e-5 * float(ref.abs().max())
        ab, wb = a.bfloat16(), w.bfloat16()
        d_a, d_w, ref = ab.cuda(), wb.cuda(), want(ab, wb)
        for product in (gemm_skinny, gemm_tc):
            out = torch.empty(M, N, dtype=torch.bfloat16, device="cuda")
            assert product(d_a, d_w, out, out_kind=2, glu=GELU_TANH)
            torch.cuda.synchronize()
            assert float((out.cpu().double() - ref).abs().max()) <= 2.0 ** -7 * float(ref.abs().max()), product.__name__


def test_a_shared_expert_beside_a_router(tmp_path):
    """The shared expert goes with any choice of experts: a pre-norm block with a softmax router and a shared expert, a
    prompt and single tokens against each other and against the same layer computed in torch."""
    from transformer_b200.architectures.generic import plan_from_spec
    from transformer_b200.engine import Engine
    from transformer_b200.parts.spec import LayerSpec, ModelSpec, PartSpec, RunEntry
    from transformer_b200.weights.random_init import random_device_weights
    d, E, k, di, sh, V = 64, 4, 2, 48, 40, 60
    norm = PartSpec.of("rmsnorm", width=d, eps=1e-6)
    att = PartSpec.of("attention", width=d, nh=2, nkvh=1, dh=32, position=PartSpec.of("rope", dh=32, theta=1e4, positions=256))
    ff = PartSpec.of("moe", width=d, di=di, nexp=E, nexp_use=k, shared_di=sh)
    spec = ModelSpec(width=d, vocab=V, max_context=256, layers=(LayerSpec(att, ff, norm, norm),), order=(RunEntry(0),),
                     embedding=PartSpec.of("lookup", vocab=V, width=d), final_norm=norm,
                     head=PartSpec.of("linear", vocab=V, width=d, tied=False))
    dev = torch.device("cuda:0")
    rules = plan_from_spec(spec)
    weights = random_device_weights(rules, 3, torch.float32, dev, 0.3)
    engine = Engine(spec, weights, torch.float32, dev, max_tokens=512)
    tokens = random_prompts(V, [70], 1)[0]
    whole = engine.step([engine.open()], [tokens], [list(range(70))]).cpu()
    slot = engine.open()
    engine.step([slot], [tokens[:60]])
    for p in range(60, 70):
        assert float((engine.step([slot], [[tokens[p]]]).cpu()[0] - whole[p]).abs().max()) < 1e-3
    seen = {}
    part = engine.layers[0].feed_forward
    x = torch.randn(9, d, generator=torch.Generator().manual_seed(5))

    class Ctx:
        tok_ids = None
        decode = False

        def scratch(self, name, shape, dtype, zero=False):
            return seen.setdefault(name, torch.zeros(shape, dtype=dtype, device=dev))

        def record(self, *a):
            pass
    got = part.forward(Ctx(), x.cuda(), None)
    out = torch.empty(9, d, device=dev)
    from transformer_b200.parts.feed_forward import sum_weighted_rows
    sum_weighted_rows(got, out)
    W = {n: t.double().cpu() for n, t in part.weights.items()}
    want = torch.zeros(9, d, dtype=torch.float64)
    for t in range(9):
        h = x[t].double()
        top = torch.topk(W["router"] @ h, k)
        for a, e in zip(torch.softmax(top.values, 0), top.indices.tolist()):
            want[t] += a * (W["wd"][e] @ (FP.silu(W["wgu"][e, :di] @ h) * (W["wgu"][e, di:] @ h)))
        s = W["shared_wd"] @ (FP.silu(W["shared_wgu"][:sh] @ h) * (W["shared_wgu"][sh:] @ h))
        want[t] += torch.sigmoid(W["shared_gate"][0] @ h) * s
    assert float((out.cpu().double() - want).abs().max()) <= 1e-4 * float(want.abs().max())
