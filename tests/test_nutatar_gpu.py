"""The Nutatar decoder on the GPU against the plain implementation
(``plain_nutatar``): each mechanism alone; whole prompts, token-by-token decoding,
portions down to two tokens, mixed batches with pages and state slots used again,
long decoding; keys far away, at page borders and on both sides of a window's
edge made to stand out, with a sink in the denominator; the first tokens of a
sequence; sizes that are 1 or equal; layers that read another layer's latents;
layers without a feed-forward; greedy generation through the engine.

bfloat16 runs use models whose routers choose far from close calls (a token's
code in a few columns of the stream that no layer writes over), so that rounding
moves logits and never an expert; float32 runs use free routers."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_nutatar as pn
from helpers import (ROOT, TOL, compare_trace, peak_tokens, random_tokens, run_trace_inprocess,
                     run_trace_subprocess, trace_mixed, trace_portions, trace_tail, trace_whole)
from nutatar_cases import CASES, PAGE_SIZES, make_folder, random_case

pytestmark = pytest.mark.gpu
DEV = torch.device("cuda:0")
DTYPES = ["float32", "bfloat16"]
LENGTHS = {"A": [31, 45, 1, 2, 90, 17], "B": [23, 60, 3, 1, 41, 8], "C": [130, 75, 2, 200, 33, 64],
           "D": [150, 3, 67, 1, 40, 270]}
NAMES = ["A", "B", "C", "D", "Asharp", "Csharp"]
# The test models are made so that a wrong key shows; rounding shows with it.
F32_SLACK = 3


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for i, (name, cfg) in enumerate(CASES.items()):
        folder = make_folder(str(tmp_path_factory.mktemp(f"ntt{name}")), cfg, seed=51 + i)
        out[name, "float32"] = (folder, pn.Plain(folder))
        folder = make_folder(str(tmp_path_factory.mktemp(f"nttb{name}")), cfg, seed=61 + i, steady=True)
        out[name, "bfloat16"] = (folder, pn.Plain(folder))
        if name in ("A", "C"):
            sharp = make_folder(str(tmp_path_factory.mktemp(f"nttsharp{name}")), cfg, seed=71 + i, sharpen=6.0)
            out[name + "sharp", "float32"] = (sharp, pn.Plain(sharp))
    return out


def sequences(name):
    key = name.replace("sharp", "")
    return {f"r{i}": random_tokens(n, CASES[key]["vocab"], 100 * i + n) for i, n in enumerate(LENGTHS[key])}


def replay(models, name, dtype, steps, tmp_path, max_tokens=None):
    folder, plain = models[name, dtype]
    out = run_trace_inprocess(folder, dtype, steps, str(tmp_path / "out"), max_tokens or peak_tokens(steps),
                              PAGE_SIZES[name.replace("sharp", "")])
    return out, plain


def names_for(dtype):
    # (where attention is peaked, bfloat16 rounding of a score is multiplied on its way to the logits)
    return NAMES if dtype == "float32" else ["A", "B", "C", "D"]


def compare(steps, out, seqs, plain, dtype, name, slack=1):
    """float32: every position within the tolerance.  bfloat16: a sub-layer's result is normed to size one
    however small it was, so the rounding of a result that nearly cancels is multiplied, and single positions
    may lie far off while the run is right (bfloat16 operands and results of the products alone, in an
    otherwise exact model, do the same at the same positions): at most one position in ten beyond the
    tolerance, none beyond ten times it, the median at most half of it."""
    if dtype == "float32":
        return compare_trace(steps, out, seqs, plain, TOL[dtype] * F32_SLACK * (3 if "sharp" in name else 1) * slack)
    compare_trace(steps, out, seqs, plain, 10 * TOL[dtype])
    fed, errs = {rid: 0 for rid in seqs}, []
    for s in steps:
        row = 0
        for e in s["entries"]:
            for w in e.get("want", []):
                ref = plain.logits(seqs[e["id"]])[fed[e["id"]] + w].numpy()
                errs.append(float(np.abs(out[s["step"]][row] - ref).max() / np.abs(ref).max()))
                row += 1
            fed[e["id"]] += len(e["tokens"])
        for rid in s.get("end", []):
            fed[rid] = 0
    errs = np.sort(np.array(errs))
    over = int((errs > TOL[dtype] * slack).sum())
    summary = f"{len(errs)} positions, median {np.median(errs):.3e}, worst {errs[-1]:.3e}, {over} beyond the tolerance"
    assert over <= max(1, len(errs) // 10) and np.median(errs) <= TOL[dtype] / 2 * slack, summary


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
@pytest.mark.parametrize("seed", [2, 3, 5, 8, 13, 34])
def test_configurations_drawn_at_random(seed, dtype, tmp_path):
    """Sizes, orders and constants nobody chose by hand: mixed batches with pages and slots used again,
    then a long tail decoded token by token."""
    cfg = random_case(seed)
    folder = make_folder(str(tmp_path / "m"), cfg, seed=seed, steady=dtype == "bfloat16")
    plain = pn.Plain(folder)
    seqs = {f"r{i}": random_tokens(n, cfg["vocab"], 31 * i + n) for i, n in enumerate([150, 70, 2, 19 + seed, 129, 1])}
    steps = trace_mixed(seqs, max_live=4, seed=seed)
    steps += trace_tail("r0", seqs["r0"], 140, step0=len(steps))
    out = run_trace_inprocess(folder, dtype, steps, str(tmp_path / "out"), max(peak_tokens(steps), 256), 16)
    compare(steps, out, seqs, plain, dtype, "random")


@pytest.mark.parametrize("dtype", DTYPES)
def test_cutting_and_batching_change_logits_by_rounding_only(models, dtype, tmp_path):
    folder, _ = models["D", dtype]
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


def launch_early(on):
    """Programmatic dependent launch in every loaded kernel library."""
    from infernum_b200.csrc import build
    for lib in build._loaded.values():
        if hasattr(lib, "ib_set_pdl"):
            lib.ib_set_pdl(1 if on else 0)


@pytest.mark.parametrize("name", list(CASES))
def test_kernels_that_start_under_their_predecessors_read_nothing_too_early(models, name, tmp_path):
    """The same steps with every kernel launched strictly after the one before it: the same bits."""
    folder, _ = models[name, "bfloat16"]
    seqs = sequences(name)
    steps = trace_mixed(seqs, max_live=4, seed=7)
    steps += trace_tail("r0", seqs["r0"], len(seqs["r0"]) - 2, step0=len(steps))
    runs = []
    try:
        for i, early in enumerate((True, True, False)):
            launch_early(early)
            runs.append(run_trace_inprocess(folder, "bfloat16", steps, str(tmp_path / f"o{i}"), peak_tokens(steps), PAGE_SIZES[name]))
    finally:
        launch_early(True)
    for other in runs[:2]:
        for step, rows in runs[2].items():
            assert np.array_equal(rows, other[step]), step


def test_the_stream_after_every_layer(models):
    """In 32-bit the stream after each layer equals the plain one."""
    from infernum_b200.cache import CacheManager
    from infernum_b200.engine.step import ModelRunner, StepEntry
    from infernum_b200.loading import load_model
    for name in CASES:
        folder, plain = models[name, "float32"]
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
        _, want = pn.forward(seq, plain.cfg, plain.weights, keep_layers=True)
        runner.step([StepEntry(cache.admit("x"), seq, [])])
        runner.check_errors()
        assert len(seen) == len(want) == len(plain.cfg["layers"])
        for i, (got, ref) in enumerate(zip(seen, want)):
            assert rel_err(got, ref) < 2e-5, f"case {name} layer {i}"


def test_the_program_itself_in_a_subprocess(models, tmp_path):
    seqs = {k: v for k, v in sequences("A").items() if len(v) > 3}
    steps = trace_mixed(seqs, max_live=3, seed=3)
    for dtype in DTYPES:
        folder, plain = models["A", dtype]
        out = run_trace_subprocess(folder, dtype, steps, str(tmp_path / dtype), peak_tokens(steps))
        compare(steps, out, seqs, plain, dtype, "A")


# ---- generation through the engine -----------------------------------------------------
def check_greedy(plain, prompt, got, dtype):
    """Every generated token is the plain implementation's best, or within rounding of it (bfloat16: at
    nine tokens of ten, see ``compare``); after a near-tie the two may part, so the comparison follows what
    was generated."""
    seq = list(prompt) + list(got)
    logits = plain.logits(seq)[len(prompt) - 1: -1]
    gaps = [float((row[pn.argmax(row)] - row[tok]) / row.abs().max()) for row, tok in zip(logits, got)]
    if dtype == "float32":
        assert max(gaps) < 1e-4, gaps
    else:
        assert sum(g > 5e-2 for g in gaps) <= max(1, len(gaps) // 10) and max(gaps) < 0.4, gaps


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(CASES))
def test_greedy_generation_through_the_engine(models, name, dtype):
    import infernum_b200 as ib
    folder, plain = models[name, dtype]
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
def test_long_generation_past_windows_from_recordings(models, dtype):
    """Replayed decode steps: windows move and states are carried under the recording."""
    import infernum_b200 as ib
    folder, plain = models["C", dtype]
    model = ib.load_model(folder, dtype=dtype)
    engine = ib.Engine(model, ib.BatchConfig(max_batch_size=2, block_size=16, num_blocks=32, max_prefill_tokens=32))
    prompts = [random_tokens(n, CASES["C"]["vocab"], 5 * n) for n in (45, 12)]
    outs = engine.generate_batch(prompts, ib.GenerateOptions(max_new_tokens=120))
    for prompt, got in zip(prompts, outs):
        assert len(got) == 120
        check_greedy(plain, prompt, got, dtype)


def test_generation_with_too_few_pages_preempts_and_recomputes(models):
    import infernum_b200 as ib
    folder, plain = models["A", "float32"]
    model = ib.load_model(folder, dtype="float32")
    engine = ib.Engine(model, ib.BatchConfig(max_batch_size=4, block_size=4, num_blocks=34, max_prefill_tokens=16))
    prompts = [random_tokens(n, CASES["A"]["vocab"], 11 * n) for n in (20, 33, 25, 14)]
    outs = engine.generate_batch(prompts, ib.GenerateOptions(max_new_tokens=30))
    for prompt, got in zip(prompts, outs):
        check_greedy(plain, prompt, got, "float32")


def test_command_line_generate(models, tmp_path):
    """``bin/generate`` picks the architecture by config.json: from a model folder, and from a bare
    configuration with random weights."""
    folder, plain = models["B", "float32"]
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

    def __init__(self, rows_per_entry, starts=None, slots=None):
        i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=DEV)  # noqa: E731
        cu = [0]
        for n in rows_per_entry:
            cu.append(cu[-1] + n)
        starts = starts or [0] * len(rows_per_entry)
        self.n_entries, self.n_rows = len(rows_per_entry), cu[-1]
        self.max_rows_per_entry = max(rows_per_entry)
        self.max_kv_len = max(s + n for s, n in zip(starts, rows_per_entry))
        self.host_cu_rows = cu
        self.scratch = {}
        self.cu_rows, self.q_start = i32(cu), i32(starts)
        self.slot_ids = i32(slots if slots is not None else list(range(self.n_entries)))
        self.row_entry = i32([e for e, n in enumerate(rows_per_entry) for _ in range(n)])
        self.positions = i32([s + i for s, n in zip(starts, rows_per_entry) for i in range(n)])


def build_pools(parts, page_size, dtype, seed, lowest=None):
    """Pools [pages, G, page_size, .] (one per item of ``parts``: per request [T, G, .]) filled through block
    tables whose pages lie in no order; NaN where nothing was written.  ``lowest``: per request the first
    position still held; pages that lie wholly before it are not there (-1)."""
    rng = np.random.default_rng(seed)
    lens = [t.shape[0] for t in parts[0]]
    need = [-(-t // page_size) for t in lens]
    pages = sum(need) + 3
    order = rng.permutation(pages - 1).tolist()
    pools = [torch.full((pages, p[0].shape[1], page_size, p[0].shape[2]), float("nan"), dtype=dtype) for p in parts]
    tables = torch.full((len(lens), max(need)), -1, dtype=torch.int32)
    for r, t in enumerate(lens):
        for b in range(need[r]):
            if lowest is not None and (b + 1) * page_size <= lowest[r]:
                continue
            page = order.pop()
            tables[r, b] = page
            n = min(page_size, t - b * page_size)
            for pool, part in zip(pools, parts):
                pool[page, :, :n] = part[r][b * page_size: b * page_size + n].transpose(0, 1).to(dtype)
    return [p.to(DEV) for p in pools], tables.to(DEV)


def latent_reference(q, kv, rank, scale, sink, gate):
    """One sequence in latent space: q [T, H, width], kv [T, width] -> [T, H, rank]."""
    T, H = q.shape[:2]
    see = pn.visible(T, None)
    out = []
    for a in range(H):
        s = q[:, a] @ kv.T * scale
        p = pn.softmax_beside(s, see, sink[a] if sink is not None else torch.tensor(float("-inf")))
        out.append(p @ kv[:, :rank] * (torch.sigmoid(gate[:, a: a + 1]) if gate is not None else 1.0))
    return torch.stack(out, dim=1)


def check_latent(dtype, H, rank, rot, page, lens, rows, run, tol, bare=False):
    """The last ``rows`` of every sequence are one step's entries.  For a sequence's last query one key is made
    to stand out beside hundreds of others: the first of all, one in the middle, a page's last and first place,
    the query's own; the sinks of some heads are as large as that key's score, others negligible."""
    g = torch.Generator().manual_seed(H * rank + rot)
    width = rank + rot
    scale = 0.5 * width ** -0.5
    r = lambda *s: torch.randn(*s, generator=g).to(dtype).double()  # noqa: E731
    qs, kvs = [r(t, H, width) for t in lens], [r(t, width) for t in lens]
    gates = None if bare else [r(t, H) * 2 for t in lens]
    sink = None if bare else torch.tensor([[-20.0, 1.0, 6.0, 0.0][h % 4] for h in range(H)]).double()
    for n, t in enumerate(lens):
        last = t - 1
        at = [0, last // 2, last // page * page, last // page * page - 1, last, 1][n % 6]
        if 0 <= at < t:
            kvs[n][at] = (qs[n][last, n % H] * (14.0 / (scale * float((qs[n][last, n % H] ** 2).sum())))).to(dtype).double()
    (pool,), tables = build_pools([[kv[:, None] for kv in kvs]], page, dtype, seed=rank)
    step = Step(rows, [t - n for t, n in zip(lens, rows)])
    pick = lambda xs: torch.cat([x[t - n:] for x, t, n in zip(xs, lens, rows)])  # noqa: E731
    q_abs = torch.empty(H, step.n_rows, width, dtype=dtype, device=DEV)
    q_abs.copy_(pick(qs).transpose(0, 1).to(dtype))
    gate = None
    if not bare:
        wide = torch.full((step.n_rows, H + 5), float("nan"), dtype=dtype, device=DEV)
        wide[:, 3: 3 + H] = pick(gates).to(dtype).to(DEV)
        gate = wide[:, 3: 3 + H]
    ref = torch.cat([latent_reference(q, kv, rank, scale, sink, z)[t - n:] for q, kv, z, t, n in
                     zip(qs, kvs, gates or [None] * len(lens), lens, rows)])
    out = torch.full((H, step.n_rows, rank), float("nan"), dtype=dtype, device=DEV)
    run(q_abs.transpose(0, 1), pool, out.transpose(0, 1), step, tables, scale,
        sink.float().to(DEV) if sink is not None else None, gate)
    assert rel_err(out.transpose(0, 1), ref) < tol


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,rank,rot,page", [(4, 24, 6, 4), (1, 8, 2, 8), (7, 64, 32, 16), (16, 300, 20, 16), (3, 33, 0, 32)])
def test_latent_attention_with_sinks_and_head_gates(dtype, H, rank, rot, page):
    from infernum_b200.ops import core
    rt = runtime(dtype)

    def run(q, pool, out, step, tables, scale, sink, gate):
        core.attention_latent_plain(q, pool, out, rank, step.positions, step.row_entry, tables, scale, 0, rt.err,
                                    sink=sink, gate=gate)

    lens = [1, 2, page, page + 1, 5 * page - 1, 201, 130]
    rows = [min(t, 5) for t in lens]
    for bare in (False, True):
        check_latent(dtype, H, rank, rot, page, lens, rows, run, 2e-5 if dtype == torch.float32 else 1e-2, bare)
    assert int(rt.err.item()) == 0


@pytest.mark.parametrize("H,rank,rot,page", [(4, 32, 16, 4), (1, 64, 32, 8), (12, 160, 16, 16), (16, 128, 64, 16), (5, 512, 64, 32)])
def test_latent_attention_with_sinks_and_head_gates_on_the_tensor_cores(H, rank, rot, page):
    """Whole prompts, portions behind cached keys, single rows, an entry without rows; every row count a CTA may
    have; the keys in slices whose merge knows the sink once and the gate."""
    from infernum_b200.ops import attention_latent
    rt = runtime(torch.bfloat16)

    def run(q, pool, out, step, tables, scale, sink, gate):
        assert attention_latent.run(q, pool, out, rank, step, tables, scale, 0, rt, sink=sink, gate=gate)

    lens = [1, 2, page, page + 1, 150, 301, 64, 97, 33]
    rows = [1, 2, 1, page + 1, 150, 1, 40, 0, 33]
    few = [1, 2, 1, 3, 1, 2, 1, 0, 1]
    for plan in [(1, 1), (2, 1), (3, 1), (4, 1), (1, 2), (1, 5), (2, 3), (4, 2), (1, 40), None]:
        rt.options["latent_plan"] = plan
        for r in (rows, few):
            check_latent(torch.bfloat16, H, rank, rot, page, lens, r, run, 1e-2)
    rt.options["latent_plan"] = (1, 3)
    check_latent(torch.bfloat16, H, rank, rot, page, lens, few, run, 1e-2, bare=True)
    assert int(rt.err.item()) == 0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,d,page,window", [(4, 2, 20, 4, 21), (1, 1, 16, 8, 5), (10, 5, 128, 16, 64), (8, 1, 64, 16, 0),
                                               (4, 4, 48, 32, 100), (3, 1, 10, 16, 1), (16, 4, 128, 16, 130)])
def test_window_with_one_in_the_denominator(dtype, H, G, d, page, window):
    """Keys just inside and just outside a window, at page borders, far away and at the query's own place made to
    stand out; scores so low that the one in the denominator matters; pages behind the window gone."""
    from infernum_b200.ops import attention as ops
    rt = runtime(dtype)
    g = torch.Generator().manual_seed(H * d + window)
    scale = 0.4 * d ** -0.5
    r = lambda *s: torch.randn(*s, generator=g).to(dtype).double()  # noqa: E731
    lens = [1, 2, page, page + 1, 5 * page - 1, 201, 130, 97, 330, 64]
    for rows in ([min(t, 5) for t in lens], [1] * len(lens), [1, 2, 1, page + 1, min(40, lens[4]), 150, 1, 0, 200, 64]):
        qs, ks, vs = [r(t, H, d) for t in lens], [r(t, G, d) for t in lens], [r(t, G, d) for t in lens]
        lowest = []
        for n, t in enumerate(lens):
            last = t - 1
            lowest.append(max(0, t - rows[n] - window + 1) if window and rows[n] else 0)
            w = window or last // 2 + 1
            at = [last, last - w + 1, last - w, last // page * page - 1, last - w + 1, last - w, last // page * page, 0,
                  last - w - 1, last - 1][n]
            a = n % G
            if 0 <= at < t:
                q = qs[n][last, a * (H // G)]
                ks[n][at, a] = (q * (11.0 / (scale * float((q * q).sum())))).to(dtype).double()
        (k_pool, v_pool), tables = build_pools([ks, vs], page, dtype, seed=d, lowest=lowest)
        step = Step(rows, [t - n for t, n in zip(lens, rows)])
        pick = lambda xs: torch.cat([x[t - n:] for x, t, n in zip(xs, lens, rows)])  # noqa: E731
        wide = torch.full((step.n_rows, H * d + 8), float("nan"), dtype=dtype, device=DEV)
        wide[:, : H * d] = pick(qs).reshape(-1, H * d).to(dtype).to(DEV)
        refs = []
        for q, k, v, t, n in zip(qs, ks, vs, lens, rows):
            see = pn.visible(t, window or None)
            refs.append(torch.stack([pn.softmax_beside(q[:, a] @ k[:, a // (H // G)].T * scale, see, 0.0)
                                     @ v[:, a // (H // G)] for a in range(H)], dim=1)[t - n:])
        out = torch.full((step.n_rows, H * d), float("nan"), dtype=dtype, device=DEV)
        ops.paged_attention(wide, k_pool, v_pool, out, step, tables, H, scale, window, rt,
                            sink=torch.zeros(H, device=DEV))
        assert rel_err(out, torch.cat(refs).reshape(-1, H * d)) < (2e-5 if dtype == torch.float32 else 1e-2)
    assert int(rt.err.item()) == 0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,d,rd,page", [(4, 2, 16, 8, 4), (1, 1, 12, 12, 8), (6, 3, 10, 0, 16), (8, 2, 64, 16, 16),
                                           (10, 5, 128, 48, 16), (40, 8, 128, 32, 16)])
def test_values_that_are_the_projected_keys(dtype, H, G, d, rd, page):
    """The value pages get the keys as projected, the key pages normed (over all heads at once) and rotated."""
    from infernum_b200.ops import core
    rt = runtime(dtype)
    g = torch.Generator().manual_seed(H * d + rd)
    T, start, eps, base = 23, 0, 1e-4, 300.0
    C = (H + G) * d
    x = torch.randn(T, C, generator=g)
    x *= (torch.arange(H + G).repeat_interleave(d) % 5 + 1.0)
    x[3] *= 1e-2
    x = x.to(dtype)
    qw, kw = torch.rand(H * d, generator=g) + 0.5, torch.rand(G * d, generator=g) + 0.5
    xd = x.double()
    q = pn.rotate_half(pn.rms_norm(xd[:, : H * d], qw.double(), eps).reshape(T, H, d), rd, base)
    k = pn.rotate_half(pn.rms_norm(xd[:, H * d:], kw.double(), eps).reshape(T, G, d), rd, base)
    pages = -(-T // page)
    k_pool, v_pool = (torch.full((pages + 1, G, page, d), 7.0, dtype=dtype, device=DEV) for _ in range(2))
    order = torch.randperm(pages, generator=g)
    step = Step([T], [start])
    rows = torch.full((T, C + (8 - C % 8) + 8), 3.0, dtype=dtype, device=DEV)
    rows[:, :C] = x.to(DEV)
    inv = torch.tensor([base ** (-2.0 * i / rd) for i in range(rd // 2)], dtype=torch.float32, device=DEV) if rd else None
    core.qk_row_norm_append(rows, qw.to(DEV), kw.to(DEV), eps, None, inv, rd, H, G, d, d, step.positions, step.row_entry,
                            order.to(torch.int32).view(1, -1).to(DEV), k_pool, v_pool, rt.err, value_from_key=True)
    tol = 2e-5 if dtype == torch.float32 else 1e-2
    assert rel_err(rows[:, : H * d], q.reshape(T, -1)) < tol and bool((rows[:, C:] == 3.0).all())
    at = torch.tensor([[int(order[p // page]), p % page] for p in range(T)])
    assert rel_err(k_pool.cpu()[at[:, 0], :, at[:, 1]], k) < tol
    assert torch.equal(v_pool.cpu()[at[:, 0], :, at[:, 1]], x[:, H * d:].reshape(T, G, d))
    assert int(rt.err.item()) == 0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,d,e,rank,tau", [(2, 16, 24, 8, 16.0), (1, 5, 1, 3, 1.0), (3, 48, 33, 16, 4.0), (4, 64, 128, 40, 16.0),
                                                (2, 128, 64, 100, 0.5), (1, 257, 8, 16, 2.0)])
def test_gated_linear_attention_in_portions_and_batches(dtype, heads, d, e, rank, tau):
    """Three requests cut differently, walked side by side through state slots in no order, against the token-by-token
    recurrence; decays from almost 1 to almost 0; a slot that an earlier request used is read as it was left and
    other slots stay as they are."""
    from infernum_b200.ops import scan
    rt = runtime(dtype)
    g = torch.Generator().manual_seed(heads * d + e)
    lens = [37, 20, 1]
    hk, hp = heads * d, heads * e
    w2 = (torch.randn(hk, rank, generator=g) * rank ** -0.5).to(dtype)
    bias = torch.randn(hk, generator=g) * 2
    bias[:3] = torch.tensor([40.0, -40.0, 90.0])[: min(3, hk)]
    off = (0, hk, 2 * hk, 2 * hk + hp + 5)
    width = off[3] + rank + 2
    seqs = [(torch.randn(n, width, generator=g)).to(dtype) for n in lens]
    refs = []
    for x in seqs:
        xd = x.double()
        w = {"a1": torch.eye(rank).double(), "a2": w2.double(), "a2.b": bias.double()}
        a = pn.decays(xd[:, off[3]: off[3] + rank], tau, w, "").reshape(-1, heads, d)
        q, k = (xd[:, o: o + hk].reshape(-1, heads, d) for o in off[:2])
        v = xd[:, off[2]: off[2] + hp].reshape(-1, heads, e)
        refs.append(torch.cat([pn.decayed_state(q[:, h] * d ** -0.5, k[:, h], v[:, h], a[:, h]) for h in range(heads)], dim=1))
    scale = max(float(r.abs().max()) for r in refs)
    for sizes in ([[37], [20], [1]], [[5, 2, 30], [1, 1, 18], [1]], [[1] * 37, [3, 17], [1]], [[36, 1], [19, 1], [1]]):
        slots = [2, 4, 0]
        state = torch.zeros(6, heads * d * e + 7, dtype=torch.float32, device=DEV)
        state[:, :7], state[5], state[1] = 3.0, 11.0, 11.0
        done = [0, 0, 0]
        got = [[], [], []]
        for i in range(max(len(s) for s in sizes)):
            live = [r for r in range(3) if i < len(sizes[r])]
            step = Step([sizes[r][i] for r in live], slots=[slots[r] for r in live])
            x = torch.cat([seqs[r][done[r]: done[r] + sizes[r][i]] for r in live]).to(DEV)
            out = torch.full((x.shape[0], hp), float("nan"), dtype=torch.float32, device=DEV)
            scan.gla_scan(x, *off, w2.to(DEV), bias.to(DEV), tau, state, 7, step, out, heads, d, e, rt)
            at = 0
            for r in live:
                n = sizes[r][i]
                got[r].append(out[at: at + n].cpu())
                at, done[r] = at + n, done[r] + n
        for r in range(3):
            err = float((torch.cat(got[r]).double() - refs[r]).abs().max()) / scale
            assert err < 3e-5, (sizes, r, err)
        assert bool((state[:, :7] == 3.0)[[0, 2, 3, 4]].all()) and bool((state[[1, 5]][:, 7:] == 11.0).all())
        assert bool((state[3, 7:] == 0.0).all())
    assert int(rt.err.item()) == 0


@pytest.mark.parametrize("E,top,count,keep", [(14, 4, 2, 1), (6, 6, 1, 1), (20, 3, 5, 2), (7, 1, 7, 1), (160, 5, 2, 1), (9, 3, 3, 3)])
def test_softmax_routing_within_the_best_groups(E, top, count, keep):
    """Also: weights that are not divided by their sum, groups scored by their one best expert (a group of many
    fair experts loses), equal scores (the lower index), further columns for a shared expert."""
    from infernum_b200.ops import core
    g = torch.Generator().manual_seed(E)
    N = 40
    z = torch.randn(N, E, generator=g) * 2
    z[1] = 0.0
    z[2, :] = z[2, 0]
    if count > 1:
        per = E // count
        z[3] = 1.0
        z[3, -1], z[3, -per: -1] = 1.5, -30.0  # one good expert in the last group, none beside it
    ids = torch.empty(N, top, dtype=torch.int32, device=DEV)
    wts = torch.empty(N, top, dtype=torch.float32, device=DEV)
    gate = torch.full((N, E + 2), float("nan"), dtype=torch.float32, device=DEV)
    extra = torch.empty(N, 2, dtype=torch.float32, device=DEV)
    core.moe_route_softmax_all(z.to(DEV), None, E, E, top, ids, wts, gate, extra, groups=count, keep=keep, group_top=1,
                               renorm=False)
    for n in range(N):
        want = pn.route(z[n].double(), top, count, keep)
        assert ids[n].tolist() == [e for e, _ in want], n
        assert torch.allclose(wts[n].cpu().double(), torch.stack([s for _, s in want]), rtol=1e-5)
        dense_row = torch.zeros(E + 2, dtype=torch.float64)
        for e, s in want:
            dense_row[e] = s
        dense_row[E:] = 1.0
        assert torch.allclose(gate[n].cpu().double(), dense_row, rtol=1e-5)
    assert bool((extra[:, 0] == 0).all()) and bool((extra[:, 1] == 1).all())


def part_weights(part, dtype, gain=1.5, seed=3):
    """Random weights of a part (rounded to bfloat16 so that both dtypes hold the same), as it wants them."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, ws in part.weight_specs().items():
        shape = ws.concrete_shape
        t = torch.randn(shape, generator=g) * (gain * shape[-1] ** -0.5 if len(shape) > 1 else 1.0)
        out[name] = t.bfloat16().to(dtype)
    return out


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("ff,limit,shared", [(64, 0.8, (128, 1.7)), (64, 1.2, (64, 1.2)), (32, None, (64, 0.5)), (24, 0.7, (40, None)),
                                             (48, 2.0, (80, 0.6)), (16, 0.9, None), (20, 0.5, (60, 1.0))])
def test_experts_beside_a_shared_one_with_a_limit_of_its_own(dtype, ff, limit, shared):
    """The shared expert as further columns of the experts' products (its width a multiple of theirs) and as a
    feed-forward of its own, few rows and prompts; every limit is reached."""
    from infernum_b200.parts import FEED_FORWARDS
    rt = runtime(dtype)
    D, E = 96, 6
    params = {"hidden_size": D, "expert_size": ff, "experts": E, "top": 3, "activation": "clamped_swish", "limit": limit,
              "alpha": 1.702, "prefix": "m.", "router_bias": None, "scoring": "softmax_all", "renormalize": False,
              "groups": {"count": 3, "keep": 2, "top": 1},
              "shared": {"size": shared[0], "prefix": "shared.", "gate": None, "limit": shared[1]} if shared else None}
    part = FEED_FORWARDS.get("moe")(params, rt)
    w = part_weights(part, dtype, gain=3.0)
    part.bind({k: v.to(DEV) for k, v in w.items()})
    assert bool(part.shared_runs) == bool(shared and shared[0] % ff == 0)
    mlp = {"expert": {"limit": limit}, "router": {"experts": E, "top": 3, "groups": {"count": 3, "keep": 2}},
           "shared": {"limit": shared[1]} if shared else None}
    g = torch.Generator().manual_seed(ff)
    x = torch.randn(700, D, generator=g).to(dtype)
    ref = pn.experts(x.double(), mlp, {k: v.double() for k, v in w.items()}, "m.")
    for n in (1, 9, 64, 300, 512, 700):
        assert rel_err(part.forward(x[:n].to(DEV)), ref[:n]) < (PART_TOL[dtype] if dtype == torch.float32 else 1e-2), n
    assert int(rt.err.item()) == 0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("D,ff", [(96, 176), (100, 36), (33, 7), (256, 512), (1024, 2048)])
def test_squared_relu_feed_forward(dtype, D, ff):
    from infernum_b200.parts import FEED_FORWARDS
    rt = runtime(dtype)
    part = FEED_FORWARDS.get("mlp")({"hidden_size": D, "intermediate_size": ff, "prefix": "m."}, rt)
    w = part_weights(part, dtype)
    part.bind({k: v.to(DEV) for k, v in w.items()})
    g = torch.Generator().manual_seed(ff)
    x = torch.randn(800, D, generator=g).to(dtype)
    ref = pn.squared_relu(x.double(), {k: v.double() for k, v in w.items()}, "m.")
    for n in (1, 7, 33, 64, 100, 256, 768, 800):
        assert rel_err(part.forward(x[:n].to(DEV)), ref[:n]) < (2e-5 if dtype == torch.float32 else 1e-2), n
    assert int(rt.err.item()) == 0


@pytest.mark.parametrize("T,N,K,splits", [(1, 300, 1024, 4), (16, 136, 2048, 8), (60, 300, 640, 1), (768, 520, 200, 0), (1024, 1000, 96, 0)])
def test_squared_relu_in_the_products_epilogue(T, N, K, splits):
    """Applied once, to the sum of all slices of K, never to a slice's part of it."""
    from infernum_b200.ops import gemm_tc
    g = torch.Generator().manual_seed(N)
    x, w = torch.randn(T, K, generator=g).bfloat16(), (torch.randn(N, K, generator=g) * K ** -0.5).bfloat16()
    ref = pn.squared_relu(x.double(), {"up": w.double(), "down": torch.eye(N).double()}, "")
    out = torch.full((T, N), float("nan"), dtype=torch.bfloat16, device=DEV)
    if splits:
        gemm_tc.gemm_tc(x.to(DEV), w.to(DEV), out, splits=splits, swiglu=gemm_tc.ALONE_CODES["relu2"])
    else:
        assert gemm_tc.act_route(x.to(DEV), w.to(DEV), out, "relu2")
    assert gemm_tc.error_flags(DEV) == 0
    assert rel_err(out, ref) < 6e-3


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_a_second_limit_from_a_column_on(dtype):
    from infernum_b200.ops import core
    g = torch.Generator().manual_seed(4)
    for I, block, col in ((192, 64, 128), (96, None, 32), (30, None, 7)):
        x = (torch.randn(11, 2 * I, generator=g) * 4).to(dtype)
        gate, up = (x.view(11, -1, 2, block).transpose(1, 2).reshape(11, 2, I).unbind(1) if block else x.split(I, dim=1))
        one = torch.eye(I, dtype=torch.float64)
        w = {"down": one}
        refs = []
        for limit in (0.7, 2.5):
            z = torch.zeros(I, I, dtype=torch.float64)
            w["gate"], w["up"] = torch.cat([one, z], 1), torch.cat([z, one], 1)
            refs.append(pn.expert(torch.cat([gate, up], 1).double(), limit, w, ""))
        ref = torch.cat([refs[0][:, :col], refs[1][:, col:]], dim=1)
        out = torch.empty(11, I, dtype=dtype, device=DEV)
        core.gated_act(x.to(DEV), out, "clamped_swish", block=block, limit=0.7, alpha=1.702, limit_col=col, limit2=2.5)
        assert rel_err(out, ref) < (1e-5 if dtype == torch.float32 else 1e-2)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_scaled_embedding_with_its_activation_copy(dtype):
    from infernum_b200.ops import core
    rt = runtime(dtype)
    table = torch.randn(50, 37).to(dtype)
    ids = torch.tensor([3, 0, 49, 7], dtype=torch.int32, device=DEV)
    out = torch.empty(4, 37, dtype=torch.float32, device=DEV)
    act = torch.empty(4, 37, dtype=dtype, device=DEV)
    core.embed_dual(ids, table.to(DEV), out, act, rt.err, 3.7)
    want = table[ids.cpu().long()].double() * 3.7
    assert rel_err(out, want) < 1e-6 and torch.equal(act, out.to(dtype))


# ---- mixers alone ------------------------------------------------------------------------
def check_mixer(spec, dtype, make_ref, sizes, page=4):
    """One mixer, one request in portions of ``sizes``, through a cache manager; the plain mixer on the whole."""
    from infernum_b200.cache import CacheManager
    from infernum_b200.engine.step import ModelRunner, StepEntry
    from infernum_b200.models.model import CacheNeed
    from infernum_b200.parts import MIXERS
    rt = runtime(dtype)
    part = MIXERS.get(spec.kind)(spec.params, rt)
    w = part_weights(part, dtype)
    part.bind({k: v.to(DEV) for k, v in w.items()})
    cache = CacheManager([CacheNeed(0, part.cache_spec(), part.state_spec(), None)], page_size=page, num_pages=80,
                         max_requests=2, dtype=dtype, device=DEV)

    class Stub:
        spec = type("S", (), {"vocab_size": 1 << 20})()

        def __init__(self):
            self.rt = rt

        def forward(self, ctx, caches):
            return part.forward(x[at: at + ctx.n_rows].to(DEV), ctx, caches[0])

    T = sum(sizes)
    g = torch.Generator().manual_seed(T)
    x = torch.randn(T, spec.params["hidden_size"], generator=g).to(dtype)
    runner = ModelRunner(Stub(), cache, max_rows=512, max_entries=2)
    rc, at, outs = cache.admit("r"), 0, []
    for n in sizes:
        outs.append(runner.step([StepEntry(rc, [0] * n, [])]))
        at += n
    ref = make_ref(x.double(), {k: v.double() for k, v in w.items()})
    assert rel_err(torch.cat(outs), ref) < (2e-5 if dtype == torch.float32 else 1.5e-2)
    assert int(rt.err.item()) == 0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name,layer", [("A", 0), ("A", 1), ("A", 3), ("B", 0), ("B", 1), ("B", 2), ("B", 4), ("B", 5), ("C", 0), ("C", 1),
                                        ("C", 2), ("D", 0), ("D", 1), ("D", 3), ("D", 4)])
def test_a_mixer_alone_in_one_portion_and_in_many(dtype, name, layer):
    from infernum_b200.models.nutatar import _mixer
    from infernum_b200.registry import resolve_config
    _, cfg = resolve_config(CASES[name])
    lay, raw = cfg.layers[layer], CASES[name]["layers"][layer]["mixer"]
    spec = _mixer(lay.type, lay.mixer, cfg, "x.")

    def ref(x, w):
        if lay.type == "latent_attention":
            return pn.latent_attention(x, pn.latents(x, raw, w, "x.", cfg.norm_eps), raw, w, "x.", cfg.norm_eps)
        return {"attention": pn.attention, "gla": pn.gla}[lay.type](x, raw, w, "x.", cfg.norm_eps)

    for sizes in ([70], [2, 5, 2, 30, 1, 1, 1, 28], [1] * 70):
        check_mixer(spec, dtype, ref, sizes)
