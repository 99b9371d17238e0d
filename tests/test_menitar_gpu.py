"""The Menitar decoder on the GPU against the plain implementation
(``plain_menitar``): each mechanism alone; whole prompts, token-by-token decoding,
portions down to two tokens, mixed batches with pages and slots used again, long
decoding; keys far away, at page borders and on both sides of a run's edge made
to stand out; the first tokens of a sequence; sizes that are 1 or equal; layers
without a feed-forward; greedy generation through the engine."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_menitar as pm
from helpers import (ROOT, TOL, compare_trace, peak_tokens, random_tokens, run_trace_inprocess,
                     run_trace_subprocess, trace_mixed, trace_portions, trace_tail, trace_whole)
from menitar_cases import CASES, PAGE_SIZES, make_folder, random_case

pytestmark = pytest.mark.gpu
DEV = torch.device("cuda:0")
DTYPES = ["float32", "bfloat16"]
LENGTHS = {"A": [31, 45, 1, 2, 90, 17], "B": [23, 60, 3, 1, 41, 8], "C": [130, 75, 2, 200, 33, 64],
           "D": [150, 3, 67, 1, 40, 270]}
NAMES = ["A", "B", "C", "D", "Asharp", "Csharp"]
# The test models' projections are scaled up (so that a wrong key shows); rounding is scaled with them.
F32_SLACK = 3


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for i, (name, cfg) in enumerate(CASES.items()):
        folder = make_folder(str(tmp_path_factory.mktemp(f"mnt{name}")), cfg, seed=51 + i)
        out[name] = (folder, pm.Plain(folder))
        if name in ("A", "C"):
            sharp = make_folder(str(tmp_path_factory.mktemp(f"mntsharp{name}")), cfg, seed=71 + i, sharpen=6.0)
            out[name + "sharp"] = (sharp, pm.Plain(sharp))
    return out


def sequences(name):
    key = name.replace("sharp", "")
    return {f"r{i}": random_tokens(n, CASES[key]["vocab"], 100 * i + n) for i, n in enumerate(LENGTHS[key])}


def replay(models, name, dtype, steps, tmp_path, max_tokens=None):
    folder, plain = models[name]
    out = run_trace_inprocess(folder, dtype, steps, str(tmp_path / "out"), max_tokens or peak_tokens(steps),
                              PAGE_SIZES[name.replace("sharp", "")])
    return out, plain


def names_for(dtype):
    # (where attention is peaked, bfloat16 rounding of a score is multiplied on its way to the logits)
    return NAMES if dtype == "float32" else ["A", "B", "C", "D"]


def compare(steps, out, seqs, plain, dtype, name, slack=1):
    if dtype == "float32":
        return compare_trace(steps, out, seqs, plain, TOL[dtype] * F32_SLACK * (3 if "sharp" in name else 1) * slack)
    return compare_trace(steps, out, seqs, plain, TOL[dtype] * slack)


def runtime(dtype, **options):
    from infernum_b200.ops import core
    from infernum_b200.parts.base import Runtime
    return Runtime(DEV, dtype, err=core.new_error_word(DEV), options=options)


def rel_err(got, ref):
    ref = ref.double().cpu()
    return float((got.double().cpu() - ref).abs().max() / max(ref.abs().max().item(), 1e-9))


PART_TOL = {torch.float32: 1e-5, torch.bfloat16: 2e-2}


# ---- whole models through the trace runner -------------------------------------------
@pytest.mark.parametrize("dtype,name", [(d, n) for d in DTYPES for n in names_for(d)])
def test_each_request_alone_and_whole(models, name, dtype, tmp_path):
    seqs = sequences(name)
    steps = []
    for rid, seq in seqs.items():
        steps += trace_whole(rid, seq, step0=len(steps))
    out, plain = replay(models, name, dtype, steps, tmp_path)
    compare(steps, out, seqs, plain, dtype, name)


@pytest.mark.parametrize("dtype,name", [(d, n) for d in DTYPES for n in names_for(d)])
def test_most_in_one_step_then_token_by_token(models, name, dtype, tmp_path):
    seqs = {k: v for k, v in sequences(name).items() if len(v) > 3}
    steps = []
    for rid, seq in seqs.items():
        steps += trace_tail(rid, seq, 40, step0=len(steps))
    out, plain = replay(models, name, dtype, steps, tmp_path)
    compare(steps, out, seqs, plain, dtype, name)


@pytest.mark.parametrize("dtype,name", [(d, n) for d in DTYPES for n in names_for(d)])
def test_a_prompt_token_by_token_from_its_first_token(models, name, dtype, tmp_path):
    seqs = {"r0": sequences(name)["r0"][:60]}
    steps = [{"step": i, "entries": [{"id": "r0", "tokens": [t], "want": [0]}], "end": []}
             for i, t in enumerate(seqs["r0"])]
    steps[-1]["end"] = ["r0"]
    out, plain = replay(models, name, dtype, steps, tmp_path)
    compare(steps, out, seqs, plain, dtype, name)


@pytest.mark.parametrize("dtype,name", [(d, n) for d in DTYPES for n in names_for(d)])
def test_portions_of_changing_size(models, name, dtype, tmp_path):
    seqs = {k: v for k, v in sequences(name).items() if len(v) > 3}
    steps = []
    for i, (rid, seq) in enumerate(seqs.items()):
        sizes = [[7, 2, 5, 3, 11, 2], [2, 2, 13, 4, 2, 9], [5, 17, 2, 3, 40], [2]][i % 4]
        steps += trace_portions(rid, seq, sizes, step0=len(steps))
    out, plain = replay(models, name, dtype, steps, tmp_path)
    compare(steps, out, seqs, plain, dtype, name)


@pytest.mark.parametrize("dtype,name", [(d, n) for d in DTYPES for n in names_for(d)])
def test_mixed_batches_with_pages_and_slots_used_again(models, name, dtype, tmp_path):
    seqs = sequences(name)
    steps = trace_mixed(seqs, max_live=4, seed=5)
    assert max(len(s["entries"]) for s in steps) >= 3
    peak = peak_tokens(steps)
    assert peak < sum((len(v) + 63) // 64 * 64 for v in seqs.values())
    out, plain = replay(models, name, dtype, steps, tmp_path, max_tokens=peak)
    compare(steps, out, seqs, plain, dtype, name)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "C"])
def test_long_decoding(models, name, dtype, tmp_path):
    seqs = {"long": random_tokens(230, CASES[name]["vocab"], 3)}
    steps = trace_tail("long", seqs["long"], tail=226)
    out, plain = replay(models, name, dtype, steps, tmp_path)
    compare(steps, out, seqs, plain, dtype, name)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("seed", [2, 3, 5, 8, 13, 21])
def test_configurations_drawn_at_random(seed, dtype, tmp_path):
    """Sizes, orders and constants nobody chose by hand: mixed batches with pages and slots used again,
    then a long tail decoded token by token."""
    cfg = random_case(seed)
    folder = make_folder(str(tmp_path / "m"), cfg, seed=seed)
    plain = pm.Plain(folder)
    seqs = {f"r{i}": random_tokens(n, cfg["vocab"], 31 * i + n) for i, n in enumerate([150, 70, 2, 19 + seed, 129, 1])}
    steps = trace_mixed(seqs, max_live=4, seed=seed)
    steps += trace_tail("r0", seqs["r0"], 140, step0=len(steps))
    out = run_trace_inprocess(folder, dtype, steps, str(tmp_path / "out"), max(peak_tokens(steps), 256), 16)
    compare(steps, out, seqs, plain, dtype, "random")


@pytest.mark.parametrize("dtype", DTYPES)
def test_cutting_and_batching_change_logits_by_rounding_only(models, dtype, tmp_path):
    folder, _ = models["D"]
    seqs = sequences("D")
    seq = seqs["r5"]
    runs = []
    mixed = trace_mixed(seqs, max_live=4, seed=9)
    for i, steps in enumerate([trace_whole("r5", seq), trace_portions("r5", seq, [7, 2, 5, 3, 11, 2]),
                               trace_tail("r5", seq, 60), mixed]):
        out = run_trace_inprocess(folder, dtype, steps, str(tmp_path / f"o{i}"), peak_tokens(steps) + 64, 16)
        rows, pos = {}, 0
        for s in steps:
            r = 0
            for e in s["entries"]:
                for w in e["want"]:
                    if e["id"] == "r5":
                        rows[pos + w] = out[s["step"]][r]
                    r += 1
                if e["id"] == "r5":
                    pos += len(e["tokens"])
        runs.append(rows)
    scale = max(np.abs(v).max() for v in runs[0].values())
    for other in runs[1:]:
        assert other
        for pos, row in other.items():
            assert np.abs(row - runs[0][pos]).max() / scale < (2e-5 if dtype == "float32" else 4e-2), pos


def test_the_stream_after_every_run_of_a_layer(models):
    """In 32-bit the stream after each run of a layer (a looped layer counts each time) equals the plain one."""
    from infernum_b200.cache import CacheManager
    from infernum_b200.engine.step import ModelRunner, StepEntry
    from infernum_b200.loading import load_model
    for name in CASES:
        folder, plain = models[name]
        model = load_model(folder, dtype="float32")
        cache = CacheManager(model.cache_needs(), page_size=4, num_pages=64, max_requests=2,
                             dtype=model.rt.dtype, device=model.rt.device)
        runner = ModelRunner(model, cache, max_rows=256, max_entries=2)
        seen = []
        for blk in model.layers:
            def hooked(stream, ctx, c, orig=blk.forward):
                orig(stream, ctx, c)
                stream.flush()
                seen.append(stream.residual.clone())
            blk.forward = hooked
        seq = random_tokens(50, CASES[name]["vocab"], 77)
        _, want = pm.forward(seq, plain.cfg, plain.weights, keep_layers=True)
        runner.step([StepEntry(cache.admit("x"), seq, [])])
        runner.check_errors()
        assert len(seen) == len(want) == len(pm.run_order(plain.cfg))
        for i, (got, ref) in enumerate(zip(seen, want)):
            assert rel_err(got, ref) < 2e-5, f"case {name} run {i}"


def test_the_program_itself_in_a_subprocess(models, tmp_path):
    seqs = {k: v for k, v in sequences("A").items() if len(v) > 3}
    steps = trace_mixed(seqs, max_live=3, seed=3)
    for dtype in DTYPES:
        folder, plain = models["A"]
        out = run_trace_subprocess(folder, dtype, steps, str(tmp_path / dtype), peak_tokens(steps))
        compare(steps, out, seqs, plain, dtype, "A")


# ---- generation through the engine -----------------------------------------------------
def check_greedy(plain, prompt, got, dtype):
    """Every generated token is the plain implementation's best, or within rounding of it; after
    a near-tie the two may part, so the comparison follows what was generated."""
    seq = list(prompt)
    for i, tok in enumerate(got):
        logits = plain.logits(seq)[-1]
        best = pm.argmax(logits)
        if tok != best:
            gap = float((logits[best] - logits[tok]) / logits.abs().max())
            assert gap < (1e-4 if dtype == "float32" else 5e-2), f"token {i}: {tok} against {best}, gap {gap:.4f}"
        seq.append(tok)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(CASES))
def test_greedy_generation_through_the_engine(models, name, dtype):
    import infernum_b200 as ib
    folder, plain = models[name]
    model = ib.load_model(folder, dtype=dtype)
    page = PAGE_SIZES[name]
    engine = ib.Engine(model, ib.BatchConfig(max_batch_size=3, block_size=page, num_blocks=480 // page,
                                             max_prefill_tokens=24))
    vocab = CASES[name]["vocab"]
    prompts = [random_tokens(n, vocab, 7 * n) for n in (5, 41, 18, 2, 30)]
    n_new = 30
    outs = engine.generate_batch(prompts, ib.GenerateOptions(max_new_tokens=n_new))
    for prompt, got in zip(prompts, outs):
        assert len(got) == n_new
        check_greedy(plain, prompt, got, dtype)
    # recurring steps ran from recordings: the parts take entries, slots and positions from the device
    assert model.replayable
    if engine.decoder is not None:
        assert engine.decoder.counts["replayed"] > 0
    # once more on the same engine: slots and pages that were used before
    again = engine.generate_batch(prompts[:2], ib.GenerateOptions(max_new_tokens=8))
    for prompt, got in zip(prompts[:2], again):
        check_greedy(plain, prompt, got, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_generation_across_the_edges_of_runs_from_recordings(models, dtype):
    """Replayed decode steps: where a request's run of positions begins moves under the recording."""
    import infernum_b200 as ib
    folder, plain = models["C"]
    model = ib.load_model(folder, dtype=dtype)
    engine = ib.Engine(model, ib.BatchConfig(max_batch_size=2, block_size=16, num_blocks=32, max_prefill_tokens=32))
    prompts = [random_tokens(n, CASES["C"]["vocab"], 5 * n) for n in (45, 12)]
    outs = engine.generate_batch(prompts, ib.GenerateOptions(max_new_tokens=120))
    for prompt, got in zip(prompts, outs):
        assert len(got) == 120
        check_greedy(plain, prompt, got, dtype)


def test_generation_with_too_few_pages_preempts_and_recomputes(models):
    import infernum_b200 as ib
    folder, plain = models["A"]
    model = ib.load_model(folder, dtype="float32")
    engine = ib.Engine(model, ib.BatchConfig(max_batch_size=4, block_size=4, num_blocks=34, max_prefill_tokens=16))
    prompts = [random_tokens(n, CASES["A"]["vocab"], 11 * n) for n in (20, 33, 25, 14)]
    outs = engine.generate_batch(prompts, ib.GenerateOptions(max_new_tokens=30))
    for prompt, got in zip(prompts, outs):
        check_greedy(plain, prompt, got, "float32")


def test_command_line_generate(models, tmp_path):
    """``bin/generate`` picks the architecture by config.json: from a model folder, and from a bare
    configuration with random weights."""
    folder, plain = models["B"]
    prompt = random_tokens(9, CASES["B"]["vocab"], 1)
    text = ",".join(map(str, prompt))
    proc = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "generate"), "-m", folder, text, "-n", "6",
                           "--greedy", "--dtype", "float32", "--block-size", "4"],
                          capture_output=True, text=True, timeout=900)
    assert proc.returncode == 0, proc.stderr[-3000:]
    line = [l for l in proc.stdout.splitlines() if l.startswith(text)][0]
    got = [int(t) for t in line.split()[1:]]
    assert len(got) == 6
    check_greedy(plain, prompt, got, "float32")
    cfg_path = tmp_path / "config.json"
    cfg_path.write_text(json.dumps(CASES["A"]))
    proc = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "generate"), "--config", str(cfg_path),
                           "--random-weights", "--weights-seed", "3", "1,2,3", "-n", "4", "--greedy",
                           "--block-size", "8"], capture_output=True, text=True, timeout=900)
    assert proc.returncode == 0, proc.stderr[-3000:]
    assert "Generated 4 tokens" in proc.stdout


# ---- mechanisms alone ------------------------------------------------------------------
class Step:
    """The device tensors of a step that the kernels read."""

    def __init__(self, rows_per_entry, starts=None):
        i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=DEV)  # noqa: E731
        cu = [0]
        for n in rows_per_entry:
            cu.append(cu[-1] + n)
        starts = starts or [0] * len(rows_per_entry)
        self.n_entries, self.n_rows = len(rows_per_entry), cu[-1]
        self.max_rows_per_entry = max(rows_per_entry)
        self.max_kv_len = max(s + n for s, n in zip(starts, rows_per_entry))
        self.cu_rows = i32(cu)
        self.row_entry = i32([e for e, n in enumerate(rows_per_entry) for _ in range(n)])
        self.positions = i32([s + i for s, n in zip(starts, rows_per_entry) for i in range(n)])


def build_pools(keys, values, page_size, dtype, seed, lowest=None):
    """Pools [pages, G, page_size, .] filled through block tables whose pages lie in no order; NaN where
    nothing was written.  ``keys`` / ``values``: per request [T, G, .].  ``lowest``: per request the first
    position still held; pages that lie wholly before it are not there (-1)."""
    rng = np.random.default_rng(seed)
    need = [-(-k.shape[0] // page_size) for k in keys]
    pages = sum(need) + 3
    order = rng.permutation(pages - 1).tolist()
    G, kw, vw = keys[0].shape[1], keys[0].shape[2], values[0].shape[2]
    k_pool = torch.full((pages, G, page_size, kw), float("nan"), dtype=dtype)
    v_pool = torch.full((pages, G, page_size, vw), float("nan"), dtype=dtype)
    tables = torch.full((len(keys), max(need)), -1, dtype=torch.int32)
    for r, (k, v) in enumerate(zip(keys, values)):
        for b in range(need[r]):
            if lowest is not None and (b + 1) * page_size <= lowest[r]:
                continue
            page = order.pop()
            tables[r, b] = page
            n = min(page_size, k.shape[0] - b * page_size)
            k_pool[page, :, :n] = k[b * page_size: b * page_size + n].transpose(0, 1).to(dtype)
            v_pool[page, :, :n] = v[b * page_size: b * page_size + n].transpose(0, 1).to(dtype)
    return k_pool.to(DEV), v_pool.to(DEV), tables.to(DEV)


def plain_talk(q, k, v, scale, temp, talk, gate, chunk, window=0):
    """One sequence: q [T, H, d], k [T, G, d], v [T, G, e], gate [T, H] -> [T, H * e]."""
    T, H = q.shape[:2]
    G = k.shape[1]
    see = pm.visible(T, chunk or None)
    if window:
        i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
        see = see & (i - j < window)
    if talk is None:
        talk = torch.eye(H, dtype=torch.float64)
    p = pm.softmax_over(pm.mixed_scores(q, k, scale, temp if temp is not None else torch.ones(H, dtype=torch.float64), talk), see)
    o = torch.stack([p[a] @ v[:, a // (H // G)] for a in range(H)], dim=1)
    if gate is not None:
        o = o * torch.sigmoid(gate)[:, :, None]
    return o.reshape(T, -1)


def check_talk(dtype, H, G, d, e, page, chunk, lens, rows, run, tol, window=0, bare=False):
    """Queries at the ends of sequences of several lengths (the last ``rows`` of each are one step's entries).
    For every sequence's last query one key is scaled so that one head's score of it stands out: the first and
    the last of the run before (which must not be seen), the run's first, one in its middle, the query's own
    neighbour, a page's first and last place.  Pages of earlier runs are gone."""
    g = torch.Generator().manual_seed(H * d + e)
    scale = 0.3 / d ** 0.5
    temp = None if bare else (0.5 + torch.rand(H, generator=g)).double()
    talk = None if bare else (torch.randn(H, H, generator=g) * H ** -0.5).bfloat16().double()
    r = lambda *s: torch.randn(*s, generator=g).to(dtype).double()  # noqa: E731
    qs, ks, vs = [r(t, H, d) for t in lens], [r(t, G, d) for t in lens], [r(t, G, e) for t in lens]
    gates = None if bare else [r(t, H) * 2 for t in lens]
    lowest = []
    for n, t in enumerate(lens):
        last = t - 1
        run0 = last // chunk * chunk if chunk else 0
        first_row = t - rows[n]
        lowest.append(max(first_row // chunk * chunk if chunk else 0, first_row - window + 1 if window else 0))
        places = [run0, run0 - 1, (run0 + last) // 2, last, run0 - chunk, last // page * page, last // page * page - 1,
                  last - window if window else 0, last - window + 1 if window else last // 3]
        at = places[n % len(places)]
        if 0 <= at < t:
            # one head's key along that query: its score stands out by some units of every other score
            a = n % G
            ks[n][at, a] = (qs[n][last, a * (H // G)] * (40.0 * d ** 0.5 / d)).to(dtype).double()
    k_pool, v_pool, tables = build_pools(ks, vs, page, dtype, seed=e, lowest=lowest)
    step = Step(rows, [t - n for t, n in zip(lens, rows)])
    pick = lambda xs: torch.cat([x[t - n:] for x, t, n in zip(xs, lens, rows)])  # noqa: E731
    wide = torch.full((step.n_rows, H * d + H + 8 - H % 8), float("nan"), dtype=dtype, device=DEV)
    # (what scales scores is in the queries: rounded once, scaled)
    factor = scale * (temp if temp is not None else torch.ones(H, dtype=torch.float64))
    qs = [(q * factor[None, :, None]).to(dtype).double() for q in qs]
    scale, temp = 1.0, None
    wide[:, : H * d] = pick(qs).reshape(-1, H * d).to(dtype).to(DEV)
    gate = None
    if not bare:
        wide[:, H * d: H * d + H] = pick(gates).to(dtype).to(DEV)
        gate = wide[:, H * d: H * d + H]
    ref = torch.cat([plain_talk(q, k, v, scale, temp, talk, z, chunk, window)[t - n:] for q, k, v, z, t, n in
                     zip(qs, ks, vs, gates or [None] * len(lens), lens, rows)])
    out = torch.full((step.n_rows, H * e + 16), float("nan"), dtype=dtype, device=DEV)
    f32 = lambda x: None if x is None else x.float().to(DEV).contiguous()  # noqa: E731
    run(wide, k_pool, v_pool, out[:, : H * e], step, tables, f32(talk), gate, chunk, window)
    assert torch.isfinite(out[:, : H * e]).all() and torch.isnan(out[:, H * e:]).all()
    assert rel_err(out[:, : H * e], ref) < tol


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,d,e,page,chunk", [(4, 2, 16, 24, 4, 21), (1, 1, 12, 12, 8, 5), (6, 3, 8, 80, 16, 64),
                                                (8, 1, 32, 64, 16, 0), (2, 2, 64, 130, 32, 100), (3, 1, 10, 5, 16, 1),
                                                (32, 8, 128, 128, 16, 48)])
def test_exchanged_scores_with_one_key_that_stands_out(dtype, H, G, d, e, page, chunk):
    from infernum_b200.ops import core
    rt = runtime(dtype)

    def run(q, k_pool, v_pool, out, step, tables, *consts):
        core.attention_talk(q, k_pool, v_pool, out, step, tables, H, *consts, rt.err)

    lens = [1, 2, page, page + 1, 5 * page - 1, 201, 64, 97, 130]
    rows = [min(t, 5) for t in lens]
    tol = 2e-5 if dtype == torch.float32 else 2e-2
    check_talk(dtype, H, G, d, e, page, chunk, lens, rows, run, tol)
    check_talk(dtype, H, G, d, e, page, chunk, lens, rows, run, tol, window=37)
    check_talk(dtype, H, G, d, e, page, chunk, lens, rows, run, tol, bare=True)
    assert int(rt.err.item()) == 0


@pytest.mark.parametrize("H,G,d,e,page,chunk", [(4, 2, 16, 32, 4, 21), (1, 1, 16, 16, 8, 5), (6, 3, 48, 80, 16, 64),
                                                (8, 1, 32, 64, 16, 0), (10, 5, 64, 128, 32, 100), (3, 1, 16, 16, 16, 1),
                                                (32, 8, 128, 128, 16, 200), (16, 4, 128, 128, 16, 32), (12, 12, 80, 96, 16, 33),
                                                (24, 4, 64, 256, 16, 50), (40, 8, 32, 32, 16, 70)])
def test_exchanged_scores_on_the_tensor_cores(H, G, d, e, page, chunk):
    """The same through the tensor-core kernel: whole prompts that fill several row tiles, portions behind
    cached keys, single decoded rows far into a sequence, an entry without rows in the middle; then the
    keys in slices over CTAs."""
    from infernum_b200.ops import attention_talk
    rt = runtime(torch.bfloat16)
    assert attention_talk.supported(H, G, d, e)

    def run(q, k_pool, v_pool, out, step, tables, *consts):
        assert attention_talk.run(q, k_pool, v_pool, out, step, tables, H, *consts, rt)

    lens = [1, 2, page, page + 1, 150, 301, 64, 97, 33, 230, 129]
    rows = [1, 2, 1, page + 1, 150, 1, 40, 0, 33, 9, 7]
    rt.options["talk_splits"] = 1
    check_talk(torch.bfloat16, H, G, d, e, page, chunk, lens, rows, run, 2e-2)
    check_talk(torch.bfloat16, H, G, d, e, page, chunk, lens, rows, run, 2e-2, window=37)
    check_talk(torch.bfloat16, H, G, d, e, page, chunk, lens, rows, run, 2e-2, bare=True)
    few = [1, 2, 1, 3, 1, 8, 1, 0, 5, 7, 1]
    for splits in (2, 3, 20):
        rt.options["talk_splits"] = splits
        check_talk(torch.bfloat16, H, G, d, e, page, chunk, lens, few, run, 2e-2)
        check_talk(torch.bfloat16, H, G, d, e, page, chunk, lens, rows, run, 2e-2, window=37)
    # the variant for few rows an entry: as many as fill eight columns of a key/value head, and one
    for n in {1, attention_talk.queries_of_few(H, G)}:
        least = [min(n, t, r) if r else 0 for t, r in zip(lens, few)]
        for splits in (1, 2, 20):
            rt.options["talk_splits"] = splits
            check_talk(torch.bfloat16, H, G, d, e, page, chunk, lens, least, run, 2e-2)
            check_talk(torch.bfloat16, H, G, d, e, page, chunk, lens, least, run, 2e-2, window=37)
        check_talk(torch.bfloat16, H, G, d, e, page, chunk, lens, least, run, 2e-2, bare=True)
        rt.options["talk_few"] = 0  # and the other one on the same rows
        check_talk(torch.bfloat16, H, G, d, e, page, chunk, lens, least, run, 2e-2)
        del rt.options["talk_few"]
    rt.options["talk_few"] = 1  # and on rows that take several of its CTAs
    check_talk(torch.bfloat16, H, G, d, e, page, chunk, lens, few, run, 2e-2)
    del rt.options["talk_few"]
    del rt.options["talk_splits"]
    check_talk(torch.bfloat16, H, G, d, e, page, chunk, lens, few, run, 2e-2)
    assert int(rt.err.item()) == 0


def test_the_exchange_keeps_32_bit_scores():
    """Scores whose large parts cancel in the exchange: s_0 = r_0 - r_1 with r_0 and r_1 some hundreds and
    nearly equal.  Rounded to bfloat16 (or to two of them) on the way the difference would be lost."""
    from infernum_b200.ops import attention_talk
    rt = runtime(torch.bfloat16)
    g = torch.Generator().manual_seed(5)
    T, H, G, d, e = 60, 4, 2, 32, 32
    base = torch.randn(T, d, generator=g)
    q = torch.stack([base, base, torch.randn(T, d, generator=g), torch.randn(T, d, generator=g)], dim=1).bfloat16().double()
    q[:, 1] = (q[:, 0] + (torch.randn(T, d, generator=g).double() * 0.01)).bfloat16().double()
    k = (torch.randn(T, G, d, generator=g) * 20).bfloat16().double()
    v = torch.randn(T, G, e, generator=g).bfloat16().double()
    talk = torch.tensor([[1.0, -1, 0, 0], [0.5, -0.5, 0, 0.01], [0, 0, 0.02, 0], [1, -1, 0.01, 0]]).bfloat16().double()
    temp = torch.ones(H).double()
    ref = plain_talk(q, k, v, 1.0, temp, talk, None, 0)
    k_pool, v_pool, tables = build_pools([k], [v], 16, torch.bfloat16, seed=1)
    step = Step([T])
    out = torch.empty(T, H * e, dtype=torch.bfloat16, device=DEV)
    args = (talk.float().to(DEV).contiguous(), None, 0, 0)
    assert attention_talk.run(q.reshape(T, H * d).bfloat16().to(DEV), k_pool, v_pool, out, step, tables, H, *args, rt)
    assert rel_err(out, ref) < 2e-2


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,d,e,rd,page", [(4, 2, 16, 24, 8, 4), (1, 1, 12, 12, 12, 8), (6, 3, 10, 7, 0, 16), (8, 2, 64, 48, 16, 16),
                                             (32, 8, 128, 128, 128, 16), (40, 8, 128, 64, 32, 16), (3, 3, 40, 16, 24, 4)])
def test_norm_over_the_whole_projection_rotation_and_cache_write(dtype, H, G, d, e, rd, page):
    """Queries in place, keys and values in their pages, against norm and rotation of the whole rows; one
    row is tiny beside eps, and heads differ in size (a norm per head would show)."""
    from infernum_b200.ops import core
    rt = runtime(dtype)
    g = torch.Generator().manual_seed(H * d + rd)
    T, start, eps, base = 23, 37, 1e-5, 300.0
    C = (H + G) * d + G * e
    x = torch.randn(T, C, generator=g)
    x[:, : H * d] *= (torch.arange(H).repeat_interleave(d) + 1.0)
    x[3] *= 1e-3
    x = x.to(dtype)
    qw, kw = torch.rand(H * d, generator=g) + 0.5, torch.rand(G * d, generator=g) + 0.5
    pos = torch.arange(start, start + T)
    q_scale = torch.rand(H, generator=g) * 3
    for normed, w_dtype, scaled in ((True, torch.float32, True), (False, torch.float32, False), (True, torch.bfloat16, False)):
        qw, kw = qw.to(w_dtype), kw.to(w_dtype)
        xd = x.double()
        q, k, v = xd[:, : H * d], xd[:, H * d: (H + G) * d], xd[:, (H + G) * d:]
        if normed:
            q, k = pm.rms_norm(q, qw.double(), eps), pm.rms_norm(k, kw.double(), eps)
        q = pm.rotate_half(q.reshape(T, H, d), pos, rd, base)
        q = (q * q_scale.double()[None, :, None] if scaled else q).reshape(T, -1)
        k = pm.rotate_half(k.reshape(T, G, d), pos, rd, base)
        pages = -(-(start + T) // page)
        k_pool = torch.full((pages + 1, G, page, d), 7.0, dtype=dtype, device=DEV)
        v_pool = torch.full((pages + 1, G, page, e), 7.0, dtype=dtype, device=DEV)
        order = torch.randperm(pages, generator=g)
        tables = order.to(torch.int32).view(1, -1).to(DEV)
        step = Step([T], [start])
        rows = torch.full((T, C + (8 - C % 8) + 8), 3.0, dtype=dtype, device=DEV)
        rows[:, :C] = x.to(DEV)
        inv = torch.tensor([base ** (-2.0 * i / rd) for i in range(rd // 2)], dtype=torch.float32, device=DEV) if rd else None
        core.qk_row_norm_append(rows, qw.to(DEV) if normed else None, kw.to(DEV) if normed else None, eps,
                                q_scale.to(DEV) if scaled else None, inv, rd, H, G, d, e,
                                step.positions, step.row_entry, tables, k_pool, v_pool, rt.err)
        tol = 2e-5 if dtype == torch.float32 else 1e-2
        assert rel_err(rows[:, : H * d], q) < tol
        assert bool((rows[:, C:] == 3.0).all())
        at = torch.tensor([[int(order[p // page]), p % page] for p in pos.tolist()])
        assert rel_err(k_pool.cpu()[at[:, 0], :, at[:, 1]], k) < tol
        assert torch.equal(v_pool.cpu()[at[:, 0], :, at[:, 1]], x[:, (H + G) * d:].reshape(T, G, e))
        written = torch.zeros(pages + 1, page, dtype=torch.bool)
        written[at[:, 0], at[:, 1]] = True
        assert bool((k_pool.cpu().transpose(1, 2)[~written] == 7.0).all())
    assert int(rt.err.item()) == 0
    bad = torch.full_like(tables, -1)
    core.qk_row_norm_append(rows, None, None, eps, None, inv, rd, H, G, d, e, step.positions, step.row_entry, bad, k_pool, v_pool,
                            rt.err)
    assert int(rt.err.item()) == 2


@pytest.mark.parametrize("act_dtype,w_dtype", [(torch.float32, torch.float32), (torch.bfloat16, torch.bfloat16),
                                               (torch.bfloat16, torch.float32)])
@pytest.mark.parametrize("W", [96, 100, 33, 2048, 4096, 9216])
def test_two_norms_of_one_sum(act_dtype, w_dtype, W):
    from infernum_b200.ops import core
    g = torch.Generator().manual_seed(W)
    N, eps = 9, 1e-4
    x, delta = torch.randn(N, W, generator=g) * 3, (torch.randn(N, W, generator=g)).to(act_dtype)
    x[2] *= 1e-4
    w1, w2 = (torch.randn(W, generator=g).to(w_dtype) for _ in range(2))
    for dl in (delta, None):
        for in_place in (True, False):
            s = x.double() + (dl.double() if dl is not None else 0)
            xd = x.to(DEV)
            x_out = xd if in_place else torch.full_like(xd, float("nan"))
            o1, o2 = (torch.empty(N, W, dtype=act_dtype, device=DEV) for _ in range(2))
            core.add_rmsnorm_pair(xd, dl.to(DEV) if dl is not None else None, x_out, w1.to(DEV), w2.to(DEV), eps, o1, o2)
            assert rel_err(x_out, s) < 1e-6
            if not in_place:
                assert torch.equal(xd.cpu(), x)
            tol = 1e-5 if act_dtype == torch.float32 else 5e-3
            assert rel_err(o1, pm.rms_norm(s, w1.double(), eps)) < tol and rel_err(o2, pm.rms_norm(s, w2.double(), eps)) < tol


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("I,block", [(64, 64), (192, 64), (100, None), (40, None)])
@pytest.mark.parametrize("limit", [0.7, 7.0, None])
def test_clamped_swish(dtype, I, block, limit):
    from infernum_b200.ops import core
    g = torch.Generator().manual_seed(I)
    N = 13
    gate, up = (torch.randn(N, I, generator=g) * 4).to(dtype), (torch.randn(N, I, generator=g) * 4).to(dtype)
    x = torch.cat([gate, up], dim=1) if block is None else \
        torch.stack([gate.view(N, -1, block), up.view(N, -1, block)], dim=2).reshape(N, 2 * I)
    one = torch.eye(I, dtype=torch.float64)
    h = torch.cat([gate, up], dim=1).double()
    z = torch.zeros(I, I, dtype=torch.float64)
    ref = pm.clamped_gated(h, {"limit": limit}, {"gate": torch.cat([one, z], 1), "up": torch.cat([z, one], 1), "down": one}, "")
    wide = torch.full((N, I + 24), 5.0, dtype=dtype, device=DEV)
    core.gated_act(x.contiguous().to(DEV), wide[:, 8: 8 + I], "clamped_swish", block=block,
                   limit=float("inf") if limit is None else limit, alpha=1.702)
    assert rel_err(wide[:, 8: 8 + I], ref) < (1e-5 if dtype == torch.float32 else 1e-2)
    assert bool((wide[:, :8] == 5.0).all()) and bool((wide[:, 8 + I:] == 5.0).all())


@pytest.mark.parametrize("T", [1, 7, 33, 64, 256, 700])
@pytest.mark.parametrize("limit", [0.8, None])
def test_clamped_swish_in_the_products_epilogue(T, limit):
    """The gate/up product with the activation applied to its 32-bit accumulators, for few tokens and on
    pairs of SMs, into the second part of wider rows."""
    from infernum_b200.ops import gemm_tc
    g = torch.Generator().manual_seed(T)
    I, K = 192, 160
    x = torch.randn(T, K, generator=g).to(torch.bfloat16)
    wg, wu = ((torch.randn(I, K, generator=g) * 0.2).to(torch.bfloat16) for _ in range(2))
    w = torch.stack([wg.view(I // 64, 64, K), wu.view(I // 64, 64, K)], dim=1).reshape(2 * I, K).contiguous()
    ref = pm.clamped_gated(x.double(), {"limit": limit}, {"gate": wg.double(), "up": wu.double(),
                                                          "down": torch.eye(I, dtype=torch.float64)}, "")
    wide = torch.full((T, I + 64), 5.0, dtype=torch.bfloat16, device=DEV)
    assert gemm_tc.swiglu_route(x.to(DEV), w.to(DEV), wide[:, 64:], activation="clamped_swish",
                                act_limit=float("inf") if limit is None else limit, act_alpha=1.702)
    assert gemm_tc.error_flags(DEV) == 0
    assert rel_err(wide[:, 64:], ref) < 6e-3
    assert bool((wide[:, :64] == 5.0).all())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("W", [96, 33, 2100])
def test_sums_that_begin_a_pass(dtype, W):
    """x + what is pending + the embedding's output + the pass's vector, the embedding's output untouched."""
    from infernum_b200.parts import ENTRIES
    from infernum_b200.parts.base import ResidualStream
    rt = runtime(dtype)
    g = torch.Generator().manual_seed(W)
    part = ENTRIES.get("add_reentry")({"hidden_size": W, "passes": 3, "step": "s"}, rt)
    step = torch.randn(3, W, generator=g).to(dtype)
    part.bind({"s": step.to(DEV)})
    x0, x, delta = (torch.randn(5, W, generator=g) for _ in range(3))
    delta = delta.to(dtype)
    for number in range(3):
        for pending in (True, False):
            for fresh in (True, False):
                origin = x0.to(DEV)
                stream = ResidualStream(origin if fresh else x.to(DEV))
                stream.origin = origin
                if pending:
                    stream.push(delta.to(DEV))
                part.forward(stream, number)
                want = (x0 if fresh else x).double() + (delta.double() if pending else 0) \
                    + (x0.double() if number else 0) + step[number].double()
                assert stream.pending is None and rel_err(stream.residual, want) < 1e-6
                assert torch.equal(origin.cpu(), x0) and stream.residual.data_ptr() != origin.data_ptr()


def test_scaled_embedding():
    from infernum_b200.ops import core
    rt = runtime(torch.bfloat16)
    table = torch.randn(50, 37).to(torch.bfloat16)
    ids = torch.tensor([3, 0, 49, 7], dtype=torch.int32, device=DEV)
    out = torch.empty(4, 37, dtype=torch.float32, device=DEV)
    core.embed(ids, table.to(DEV), out, rt.err, 3.7)
    assert rel_err(out, table[ids.cpu().long()].double() * 3.7) < 1e-6


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("ff,joint", [(64, True), (36, False)])
def test_parallel_layer_in_one_closing_product_or_two(dtype, ff, joint):
    """A block of stand-in attention and feed-forward: both forms of its end give x + (mixer + feed-forward)."""
    from infernum_b200.loading import load_model  # noqa: F401  (registers the parts)
    from infernum_b200.models.model import Model
    from infernum_b200.cache import CacheManager
    from infernum_b200.engine.step import ModelRunner, StepEntry
    from infernum_b200.registry import resolve_config
    from infernum_b200.weights.random_init import random_tensors
    from menitar_cases import attention, dense
    cfg = {"architecture": "Menitar", "vocab": 90, "width": 72, "norm": {"eps": 1e-5},
           "layers": [attention(2, 1, 16, 32, 0.3, 6, (8, 100.0), dense(ff, 0.9))]}
    arch, typed = resolve_config(cfg)
    rt = runtime(dtype)
    model = Model(arch.build_spec(typed), rt)
    weights = random_tensors(model.weight_specs(), 3, DEV, dtype)
    for n in weights:
        if n.endswith((".gate", ".up", ".v", ".o", ".down")):
            weights[n] = weights[n] * 4
    model.bind(weights)
    assert (model.layers[0].joint is not None) == joint
    cache = CacheManager(model.cache_needs(), page_size=4, num_pages=16, max_requests=1, dtype=dtype, device=DEV)
    runner = ModelRunner(model, cache)
    seq = random_tokens(20, 90, 4)
    got = runner.step([StepEntry(cache.admit("a"), seq, list(range(20)))])
    runner.check_errors()
    ref = pm.forward(seq, cfg, {k: v.double().cpu() for k, v in weights.items()})
    assert rel_err(got, ref) < (2e-5 if dtype == torch.float32 else 4e-2)
