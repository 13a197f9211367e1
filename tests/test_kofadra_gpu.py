"""The Kofadra decoder in the engine against the plain implementation (plain_kofadra.py): every mechanism in a model of
its own, whole prompts, prompts against token-by-token decoding, portions down to two tokens, unequal batches against
each request alone, slots, pages and rings that are used again, decoding across page borders and every chunk's edge, the
first tokens, other sizes (one head, one stream, one expert, one tap, chunks of one position, heads that need padding,
layers without feed-forward, loops), chunks of hundreds of tokens, recorded steps, and greedy generation through the
library's own entry point."""
import pytest
import torch

import plain_kofadra as plain
import tiny_kofadra as tiny
from test_relilix_gpu import RouterSpy, check

pytestmark = pytest.mark.gpu


def routed_runs(cfg):
    """The layer runs (in the order they run) that have a routed feed-forward."""
    return [run for run, i in enumerate(plain.run_order(cfg)) if cfg["layers"][i].get("mlp")]


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    tmp = tmp_path_factory.mktemp("kofadra")
    return {name: tiny.make_folder(tmp, name, seed=90 + i) for i, name in enumerate(tiny.ALL)}


@pytest.fixture(scope="module")
def plains(folders):
    return {name: tiny.load_plain(f) for name, f in folders.items()}


_models = {}


def model_for(folders, name, dtype, **kw):
    """bfloat16 engines run without recorded steps unless asked: their checks watch which experts the router chose, and a
    replayed recording calls nothing that could be watched."""
    from catena_models_b200.api import Model

    if dtype == "bfloat16":
        kw.setdefault("use_graphs", False)
    key = (name, dtype, tuple(sorted(kw.items())))
    if key not in _models:
        _models[key] = Model.load(folders[name], dtype=dtype, max_tokens=8192, **kw)
    return _models[key]


_exact = {}


def exact(plains, name, tokens, dtype="float32", ids=None):
    """The plain logits; for bfloat16 (exact, yardstick), both with the experts `ids` ({run: [T, top]})."""
    cfg, tensors = plains[name]
    if dtype == "bfloat16":
        return (plain.forward(tokens, tensors, cfg, expert_ids=ids)[0],
                plain.forward(tokens, tensors, cfg, rd=plain.to_bf16, expert_ids=ids)[0])
    key = (name, tuple(tokens))
    if key not in _exact:
        _exact[key] = plain.forward(tokens, tensors, cfg)[0]
    return _exact[key]


def run_alone(engine, tokens, cuts, cfg=None):
    """One request through the engine in steps of the given sizes (the rest token by token); every logit.  With `cfg`:
    (logits, {run: the experts the engine chose, [T, top]})."""
    (slot,) = engine.admit(1)
    out, at = [], 0
    with RouterSpy() as spy:
        try:
            for n in list(cuts) + [1] * len(tokens):
                if at >= len(tokens):
                    break
                part = tokens[at:at + n]
                spy.begin_step()
                out.append(engine.step([slot], [part], [list(range(len(part)))]).float().cpu())
                at += len(part)
            engine.check_errors()
        finally:
            engine.release([slot])
    if cfg is None:
        return torch.cat(out)
    runs = routed_runs(cfg)
    if any(len(step) != len(runs) for step in spy.steps):
        return torch.cat(out), None                       # recorded steps: nothing was seen
    return torch.cat(out), {run: torch.cat([step[j] for step in spy.steps]) for j, run in enumerate(runs)}


def alone_against_plain(engine, plains, name, tokens, cuts, dtype):
    got, ids = run_alone(engine, tokens, cuts, plains[name][0])
    check(got, exact(plains, name, tokens, dtype, ids if dtype == "bfloat16" else None), dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", [n for n in tiny.ALL if n != "L"])
def test_whole_prompt(folders, plains, name, dtype):
    engine = model_for(folders, name, dtype).engine
    tokens = tiny.prompt(150, tiny.ALL[name]["vocab"], 1)
    alone_against_plain(engine, plains, name, tokens, [len(tokens)], dtype)


def test_the_sum_of_the_streams_after_every_layer_run(folders, plains):
    from catena_models_b200.parts.parallel import HyperBlock

    engine = model_for(folders, "A", "float32").engine
    cfg, tensors = plains["A"]
    tokens = tiny.prompt(90, cfg["vocab"], 5)
    want = []
    plain.forward(tokens, tensors, cfg, streams=want)
    got, original = [], HyperBlock.forward

    def spy(self, rt, batch, h, n, state, next_norm):
        out = original(self, rt, batch, h, n, state, next_norm)
        got.append(out[0][:len(tokens)].detach().double().sum(1).cpu())
        return out

    HyperBlock.forward = spy
    try:
        run_alone(engine, tokens, [len(tokens)])
    finally:
        HyperBlock.forward = original
    assert len(got) == len(want) == 8
    for g, w in zip(got, want):
        assert float((g - w).abs().max() / w.abs().max()) < 1e-5


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C", "M", "delta", "attention", "moe", "streams"])
def test_prompt_then_token_by_token(folders, plains, name, dtype):
    """A prompt in one step, then tokens one by one (recorded decode steps from the second on): across page borders (64,
    128), every chunk's edge and every ring's end, and from the very first token on."""
    engine = model_for(folders, name, dtype).engine
    tokens = tiny.prompt(150, tiny.ALL[name]["vocab"], 2)
    alone_against_plain(engine, plains, name, tokens, [50], dtype)
    if dtype == "float32" or name in ("A", "B"):
        alone_against_plain(engine, plains, name, tokens, [1], dtype)


@pytest.mark.parametrize("name", ["A", "B", "C", "M"])
def test_portions_of_several_sizes(folders, plains, name):
    engine = model_for(folders, name, "float32").engine
    tokens = tiny.prompt(200, tiny.ALL[name]["vocab"], 3)
    ref = exact(plains, name, tokens)
    for cuts in ([2] * 100, [3, 61, 1, 64, 2, 69], [64, 64, 64, 8], [127, 2, 2, 69], [1, 1, 2, 5, 7, 100, 84], [20, 20, 30, 50, 80]):
        check(run_alone(engine, tokens, cuts), ref, "float32")
    bf = model_for(folders, name, "bfloat16").engine
    alone_against_plain(bf, plains, name, tokens, [33, 2, 65, 100], "bfloat16")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C", "M"])
def test_unequal_batch_against_each_alone(folders, plains, name, dtype):
    """Four requests of unequal length start together and are decoded together; the shorter ones end earlier and
    their slots, pages and rings are taken by new requests while the others go on."""
    engine = model_for(folders, name, dtype).engine
    cfg = plains[name][0]
    vocab, runs = cfg["vocab"], routed_runs(cfg)
    lens, extra = [1, 70, 23, 131], [3, 9, 30, 12]
    toks = [tiny.prompt(n + e, vocab, 10 + i) for i, (n, e) in enumerate(zip(lens, extra))]
    slots = engine.admit(4)
    got = [[] for _ in toks]
    chosen = [{run: [] for run in runs} for _ in toks]          # per request and routed run: the engine's experts

    def seen(step, owners):
        """Hand a step's recorded choices to the requests that own its rows (owners: (request, rows) in row order)."""
        if len(step) != len(runs):
            return
        for j, run in enumerate(runs):
            at = 0
            for i, n in owners:
                chosen[i][run].append(step[j][at:at + n])
                at += n

    with RouterSpy() as spy:
        spy.begin_step()
        logits = engine.step(slots, [t[:n] for t, n in zip(toks, lens)], [list(range(n)) for n in lens]).float().cpu()
        seen(spy.steps[-1], list(enumerate(lens)))
        at = 0
        for i, n in enumerate(lens):
            got[i].append(logits[at:at + n])
            at += n
        live, pos = list(range(4)), list(lens)
        late = None
        while live:
            spy.begin_step()
            logits = engine.step([slots[i] for i in live], [[toks[i][pos[i]]] for i in live]).float().cpu()
            seen(spy.steps[-1], [(i, 1) for i in live])
            for r, i in enumerate(live):
                got[i].append(logits[r:r + 1])
                pos[i] += 1
            done = [i for i in live if pos[i] == len(toks[i])]
            for i in done:
                engine.release([slots[i]])
            live = [i for i in live if i not in done]
            if done and late is None and live:
                # a new request takes a slot that was just given back, while the others decode on
                late_tokens = tiny.prompt(40, vocab, 99)
                (s,) = engine.admit(1)
                assert s in [slots[i] for i in done]
                spy.begin_step()
                late = engine.step([s], [late_tokens], [list(range(40))]).float().cpu()
                late_ids = {run: spy.steps[-1][j] for j, run in enumerate(runs)} if len(spy.steps[-1]) == len(runs) else None
                engine.release([s])
    engine.check_errors()
    for i in range(4):
        ids = {run: torch.cat(chosen[i][run]) for run in runs} if dtype == "bfloat16" else None
        check(torch.cat(got[i]), exact(plains, name, toks[i], dtype, ids), dtype)
    check(late, exact(plains, name, late_tokens, dtype, late_ids if dtype == "bfloat16" else None), dtype)


@pytest.mark.parametrize("name", ["A", "M"])
def test_mixed_step_of_started_and_new_requests(folders, plains, name):
    """One step in which a started request brings several tokens, another one token and a third its whole prompt."""
    engine = model_for(folders, name, "float32").engine
    vocab = tiny.ALL[name]["vocab"]
    a, b, c = tiny.prompt(90, vocab, 31), tiny.prompt(70, vocab, 32), tiny.prompt(66, vocab, 33)
    sa, sb, sc = engine.admit(3)
    engine.step([sa, sb], [a[:60], b[:69]], [[], []])
    logits = engine.step([sa, sb, sc], [a[60:], b[69:], c], [list(range(30)), [0], list(range(66))]).float().cpu()
    engine.check_errors()
    engine.release([sa, sb, sc])
    check(logits[:30], exact(plains, name, a)[60:], "float32")
    check(logits[30:31], exact(plains, name, b)[69:], "float32")
    check(logits[31:], exact(plains, name, c), "float32")


@pytest.mark.parametrize("name", ["A", "C"])
def test_long_decoding(folders, plains, name):
    """Hundreds of single tokens: every ring turns over several times, the growing caches cross several pages."""
    engine = model_for(folders, name, "float32").engine
    tokens = tiny.prompt(330, tiny.ALL[name]["vocab"], 4)
    check(run_alone(engine, tokens, [5]), exact(plains, name, tokens), "float32")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_chunks_of_hundreds_of_tokens(folders, plains, dtype):
    """Chunks of 800 and of 333 over prompts of 1,000 tokens (the long-prompt attention kernels of the bfloat16 engine),
    then single tokens that step into the next chunk, and a portion on top of held tokens."""
    engine = model_for(folders, "L", dtype).engine
    tokens = tiny.prompt(1000, tiny.ALL["L"]["vocab"], 6)
    ref = exact(plains, "L", tokens, dtype)
    check(run_alone(engine, tokens, [970]), ref, dtype)
    check(run_alone(engine, tokens, [790, 180, 15]), ref, dtype)
    check(run_alone(engine, tokens, [650, 350]), ref, dtype)


@pytest.mark.parametrize("name", ["A", "M"])
def test_recorded_prompt_classes(folders, plains, name):
    """Prompts of one class of shapes (rows rounded up to 64, the same number of wanted places) run as a replayed
    recording from the third on, with rows of padding behind the tokens; so do portions on top of held tokens."""
    engine = model_for(folders, name, "float32").engine
    vocab = tiny.ALL[name]["vocab"]
    before = len(engine._prompt_graphs)
    got, ref = [], []
    for n in (130, 150, 170, 192, 135):
        tokens = tiny.prompt(n, vocab, 40 + n)
        (slot,) = engine.admit(1)
        got.append(engine.step([slot], [tokens], [[n - 3, n - 1]]).float().cpu())
        engine.release([slot])
        ref.append(exact(plains, name, tokens)[[n - 3, n - 1]])
    for n in (200, 230, 250, 210):
        tokens = tiny.prompt(n, vocab, 50 + n)
        (slot,) = engine.admit(1)
        engine.step([slot], [tokens[:60]], [[]])
        got.append(engine.step([slot], [tokens[60:]], [[0, n - 61]]).float().cpu())
        engine.release([slot])
        ref.append(exact(plains, name, tokens)[[60, n - 1]])
    engine.check_errors()
    assert len(engine._prompt_graphs) >= before + 2          # both classes were recorded (and then replayed)
    check(torch.cat(got), torch.cat(ref), "float32")


@pytest.mark.parametrize("name", ["A", "M", "B"])
def test_recorded_bfloat16_steps_against_unrecorded_ones(folders, name):
    """The bfloat16 engine with recorded steps (single tokens from the second step on) against the same engine without:
    the same kernels on the same rows."""
    plain_engine = model_for(folders, name, "bfloat16").engine
    recorded = model_for(folders, name, "bfloat16", use_graphs=True).engine
    tokens = tiny.prompt(180, tiny.ALL[name]["vocab"], 8)
    a, b = run_alone(plain_engine, tokens, [70]), run_alone(recorded, tokens, [70])
    assert len(recorded._graphs) >= 1
    assert float((a - b).abs().max()) <= 1e-6 * float(a.abs().max())


@pytest.mark.parametrize("name", ["A", "M"])
def test_the_recurrence_in_chunks_and_row_by_row(folders, plains, name):
    """Prompts that the delta rule takes in chunks of 64 rows (also a last chunk of one row, and chunks that begin on top of
    held tokens) give the numbers of the row-by-row walk."""
    from catena_models_b200.parts.recurrent import DeltaRule

    engine = model_for(folders, name, "float32", use_graphs=False).engine
    tokens = tiny.prompt(193, tiny.ALL[name]["vocab"], 12)
    keep = DeltaRule.CHUNKED_MIN_ROWS
    rows = {}
    try:
        for least in (1, 1 << 30):
            DeltaRule.CHUNKED_MIN_ROWS = least
            rows[least] = [run_alone(engine, tokens, cuts) for cuts in ([193], [129, 64], [2, 3, 65, 123])]
    finally:
        DeltaRule.CHUNKED_MIN_ROWS = keep
    for a, b in zip(rows[1], rows[1 << 30]):
        check(a, b, "float32")
        check(a, exact(plains, name, tokens), "float32")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_library(folders, plains, dtype):
    """Model.generate (scheduler, batches, recorded steps, on-device argmax) against greedy decoding: with the plain
    implementation in float32; in bfloat16 with the unrecorded engine's own logits for the same tokens, where a token that
    is not their best must be as good as the best within the noise of the format."""
    model = model_for(folders, "A", dtype, use_graphs=True)
    cfg, tensors = plains["A"]
    prompts = [tiny.prompt(n, cfg["vocab"], 60 + n) for n in (5, 37, 70)]
    outs = model.generate(prompts, max_new_tokens=12, temperature=0.0, ignore_eos=True)
    for p, o in zip(prompts, outs):
        new = list(o.tokens)
        assert len(new) == 12
        seq = list(p) + new
        if dtype == "float32":
            logits = plain.forward(seq, tensors, cfg)[0]
        else:
            logits = run_alone(model_for(folders, "A", dtype).engine, seq, [len(p)]).double()
        for j, tok in enumerate(new):
            row = logits[len(p) - 1 + j]
            best = int(row.argmax())
            if tok != best:
                gap = float(row[best] - row[tok]) / float(row.abs().max())
                assert dtype == "bfloat16" and gap < 0.03, (tok, best, gap)


def test_a_plain_residual_in_place_of_streams(tmp_path, plains):
    """A configuration without `streams`: the same layers on a plain float32 residual.  With one stream, read, put and mix
    factors of one, the streams compute just that."""
    import copy

    from catena_models_b200.api import Model

    cfg = copy.deepcopy(tiny.ONLY_ATTENTION)
    cfg["layers"].append(tiny.delta(2, 1, 8, 12, 3, tiny.moe(16, 4, 2)))
    tensors = tiny.make_tensors(cfg, 5)
    for name in tensors:
        if ".hc" in name:
            tensors[name] = torch.ones_like(tensors[name])
    folder = tiny.make_folder(tmp_path, "one", config=cfg, tensors=tensors)
    bare = {k: v for k, v in cfg.items() if k != "streams"}
    folder2 = tiny.make_folder(tmp_path, "bare", config=bare, tensors={k: v for k, v in tensors.items() if ".hc" not in k})
    tokens = tiny.prompt(100, cfg["vocab"], 3)
    ref = plain.forward(tokens, tiny.load_plain(folder)[1], cfg)[0]
    for f in (folder, folder2):
        check(run_alone(Model.load(f, dtype="float32", max_tokens=1024).engine, tokens, [60]), ref, "float32")


def test_command_line(folders, plains, tmp_path):
    """The library's command line on a model folder (greedy tokens against the plain statement) and on random weights
    from a configuration file (its prompt and decode timings)."""
    import json
    import os
    import subprocess
    import sys

    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfg, tensors = plains["C"]
    p1, p2 = tiny.prompt(6, cfg["vocab"], 1), tiny.prompt(13, cfg["vocab"], 2)
    cmd = [sys.executable, "-m", "catena_models_b200", "--model", folders["C"], "--dtype", "float32", "-n", "5",
           "--ignore-eos", "--prompt", " ".join(map(str, p1)), "--prompt", ",".join(map(str, p2))]
    run = subprocess.run(cmd, cwd=root, capture_output=True, text=True, timeout=600)
    assert run.returncode == 0, run.stderr
    lines = [list(map(int, l.split())) for l in run.stdout.strip().splitlines()]
    want = []
    for p in (p1, p2):
        seq = list(p)
        for _ in range(5):
            seq.append(int(plain.forward(seq, tensors, cfg)[0][-1].argmax()))
        want.append(seq[len(p):])
    assert [l[-5:] for l in lines] == want
    conf = tmp_path / "c.json"
    conf.write_text(json.dumps(tiny.TINY_M))
    bench = subprocess.run([sys.executable, "-m", "catena_models_b200", "--random", str(conf), "--bench", "--pp", "200",
                            "--tg", "6", "--tg-context", "150", "--batch", "2"], cwd=root, capture_output=True,
                           text=True, timeout=600)
    assert bench.returncode == 0, bench.stderr
    assert "pp200x2" in bench.stdout and "tg6/ctx150x2" in bench.stdout
