"""The Mogilorn decoder in the engine against the plain implementation (plain_mogilorn.py): every mechanism in a model of
its own, whole prompts, prompts against token-by-token decoding, portions down to two tokens, unequal batches against
each request alone, slots, pages and rings that are used again, decoding across page borders and every window's edge, the
first tokens, other sizes (one head, heads that need padding, windows of one position, layers without feed-forward),
windows of hundreds of tokens, recorded steps, and greedy generation through the library's own entry point."""
import copy

import pytest
import torch

import plain_mogilorn as plain
import tiny_mogilorn as tiny
from test_relilix_gpu import check as check_bfloat16
from test_relilix_gpu import row_errs

pytestmark = pytest.mark.gpu

# Largest |engine - plain| relative to the largest |logit| of the row.  Angles are float32 products: at position 330 and rates
# near one that alone moves a logit by up to 7e-5 (the plain statement with such angles against itself); a constant of the
# configuration that is off by a little moves it by 1e-3 and more (test_constants_that_must_show).
TOL_F32 = 1e-4


def check(got, ref, dtype):
    if dtype == "bfloat16":
        check_bfloat16(got, ref, dtype)
        return
    assert got.shape == ref.shape and bool(torch.isfinite(got).all())
    assert float(row_errs(got, ref).max()) < TOL_F32, float(row_errs(got, ref).max())


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    tmp = tmp_path_factory.mktemp("mogilorn")
    return {name: tiny.make_folder(tmp, name, seed=120 + i) for i, name in enumerate(tiny.ALL)}


@pytest.fixture(scope="module")
def plains(folders):
    return {name: tiny.load_plain(f) for name, f in folders.items()}


_models = {}


def model_for(folders, name, dtype, **kw):
    from catena_models_b200.api import Model

    key = (name, dtype, tuple(sorted(kw.items())))
    if key not in _models:
        _models[key] = Model.load(folders[name], dtype=dtype, max_tokens=8192, **kw)
    return _models[key]


_exact = {}


def exact(plains, name, tokens, dtype="float32"):
    """The plain logits; for bfloat16 (exact, yardstick)."""
    cfg, tensors = plains[name]
    key = (name, tuple(tokens), dtype)
    if key not in _exact:
        out = plain.forward(tokens, tensors, cfg)[0]
        _exact[key] = out if dtype == "float32" else (out, plain.forward(tokens, tensors, cfg, rd=plain.to_bf16)[0])
    return _exact[key]


def cut_rows(ref, rows):
    return tuple(r[rows] for r in ref) if isinstance(ref, tuple) else ref[rows]


def run_alone(engine, tokens, cuts):
    """One request through the engine in steps of the given sizes (the rest token by token); every logit."""
    (slot,) = engine.admit(1)
    out, at = [], 0
    try:
        for n in list(cuts) + [1] * len(tokens):
            if at >= len(tokens):
                break
            part = tokens[at:at + n]
            out.append(engine.step([slot], [part], [list(range(len(part)))]).float().cpu())
            at += len(part)
        engine.check_errors()
    finally:
        engine.release([slot])
    return torch.cat(out)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", [n for n in tiny.ALL if n != "L"])
def test_whole_prompt(folders, plains, name, dtype):
    engine = model_for(folders, name, dtype).engine
    for n in (150, 1, 3):
        tokens = tiny.prompt(n, tiny.ALL[name]["vocab"], n)
        check(run_alone(engine, tokens, [n]), exact(plains, name, tokens, dtype), dtype)


@pytest.mark.parametrize("name", ["A", "B"])
def test_the_stream_after_every_layer(folders, plains, name):
    from catena_models_b200.parts.parallel import OutputNormBlock

    engine = model_for(folders, name, "float32").engine
    cfg, tensors = plains[name]
    tokens = tiny.prompt(90, cfg["vocab"], 5)
    want = []
    plain.forward(tokens, tensors, cfg, streams=want)
    got, original = [], OutputNormBlock.forward

    def spy(self, rt, batch, h, n, state, next_norm):
        out = original(self, rt, batch, h, n, state, next_norm)
        got.append(out[0][:len(tokens)].detach().double().cpu())
        return out

    OutputNormBlock.forward = spy
    try:
        run_alone(engine, tokens, [len(tokens)])
    finally:
        OutputNormBlock.forward = original
    assert len(got) == len(want) == len(cfg["layers"])
    for g, w in zip(got, want):
        assert float((g - w).abs().max() / w.abs().max()) < 1e-5


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", [n for n in tiny.ALL if n != "L"])
def test_prompt_then_token_by_token(folders, plains, name, dtype):
    """A prompt in one step, then tokens one by one (recorded decode steps from the second on): across page borders (64,
    128), every window's edge and every ring's end, and from the very first token on."""
    engine = model_for(folders, name, dtype).engine
    tokens = tiny.prompt(150, tiny.ALL[name]["vocab"], 2)
    ref = exact(plains, name, tokens, dtype)
    check(run_alone(engine, tokens, [50]), ref, dtype)
    check(run_alone(engine, tokens, [1]), ref, dtype)


@pytest.mark.parametrize("name", ["A", "B", "C", "M", "W"])
def test_portions_of_several_sizes(folders, plains, name):
    engine = model_for(folders, name, "float32").engine
    tokens = tiny.prompt(200, tiny.ALL[name]["vocab"], 3)
    ref = exact(plains, name, tokens)
    for cuts in ([2] * 100, [3, 61, 1, 64, 2, 69], [64, 64, 64, 8], [127, 2, 2, 69], [1, 1, 2, 5, 7, 100, 84], [20, 20, 30, 50, 80]):
        check(run_alone(engine, tokens, cuts), ref, "float32")
    bf = model_for(folders, name, "bfloat16").engine
    check(run_alone(bf, tokens, [33, 2, 65, 100]), exact(plains, name, tokens, "bfloat16"), "bfloat16")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C", "M"])
def test_unequal_batch_against_each_alone(folders, plains, name, dtype):
    """Four requests of unequal length start together and are decoded together; the shorter ones end earlier and
    their slots, pages and rings are taken by new requests while the others go on."""
    engine = model_for(folders, name, dtype).engine
    vocab = plains[name][0]["vocab"]
    lens, extra = [1, 70, 23, 131], [3, 9, 30, 12]
    toks = [tiny.prompt(n + e, vocab, 10 + i) for i, (n, e) in enumerate(zip(lens, extra))]
    slots = engine.admit(4)
    got = [[] for _ in toks]
    logits = engine.step(slots, [t[:n] for t, n in zip(toks, lens)], [list(range(n)) for n in lens]).float().cpu()
    at = 0
    for i, n in enumerate(lens):
        got[i].append(logits[at:at + n])
        at += n
    live, pos, late = list(range(4)), list(lens), None
    while live:
        logits = engine.step([slots[i] for i in live], [[toks[i][pos[i]]] for i in live]).float().cpu()
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
            late = engine.step([s], [late_tokens], [list(range(40))]).float().cpu()
            engine.release([s])
    engine.check_errors()
    for i in range(4):
        check(torch.cat(got[i]), exact(plains, name, toks[i], dtype), dtype)
    check(late, exact(plains, name, late_tokens, dtype), dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "M"])
def test_mixed_step_of_started_and_new_requests(folders, plains, name, dtype):
    """One step in which a started request brings several tokens, another one token and a third its whole prompt."""
    engine = model_for(folders, name, dtype).engine
    vocab = tiny.ALL[name]["vocab"]
    a, b, c = tiny.prompt(150, vocab, 31), tiny.prompt(70, vocab, 32), tiny.prompt(66, vocab, 33)
    sa, sb, sc = engine.admit(3)
    engine.step([sa, sb], [a[:60], b[:69]], [[], []])
    logits = engine.step([sa, sb, sc], [a[60:], b[69:], c], [list(range(90)), [0], list(range(66))]).float().cpu()
    engine.check_errors()
    engine.release([sa, sb, sc])
    check(logits[:90], cut_rows(exact(plains, name, a, dtype), slice(60, None)), dtype)
    check(logits[90:91], cut_rows(exact(plains, name, b, dtype), slice(69, None)), dtype)
    check(logits[91:], exact(plains, name, c, dtype), dtype)


@pytest.mark.parametrize("name", ["A", "C"])
def test_long_decoding(folders, plains, name):
    """Hundreds of single tokens: every ring turns over several times, the growing caches cross several pages."""
    engine = model_for(folders, name, "float32").engine
    tokens = tiny.prompt(330, tiny.ALL[name]["vocab"], 4)
    check(run_alone(engine, tokens, [5]), exact(plains, name, tokens), "float32")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_windows_of_hundreds_of_tokens(folders, plains, dtype):
    """Windows of 333 and 800 over prompts of 1,000 tokens (the long-prompt attention kernels of the bfloat16 engine), then
    single tokens over rings that have turned over, and portions on top of held tokens."""
    engine = model_for(folders, "L", dtype).engine
    tokens = tiny.prompt(1000, tiny.ALL["L"]["vocab"], 6)
    ref = exact(plains, "L", tokens, dtype)
    check(run_alone(engine, tokens, [970]), ref, dtype)
    check(run_alone(engine, tokens, [790, 180, 15]), ref, dtype)
    check(run_alone(engine, tokens, [650, 350]), ref, dtype)


@pytest.mark.parametrize("name", ["A", "M"])
def test_recorded_prompt_classes(folders, plains, name):
    """Prompts of one class of shapes run as a replayed recording from the third on, with rows of padding behind the tokens;
    so do portions on top of held tokens."""
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
    plain_engine = model_for(folders, name, "bfloat16", use_graphs=False).engine
    recorded = model_for(folders, name, "bfloat16", use_graphs=True).engine
    tokens = tiny.prompt(180, tiny.ALL[name]["vocab"], 8)
    a, b = run_alone(plain_engine, tokens, [70]), run_alone(recorded, tokens, [70])
    assert len(recorded._graphs) >= 1
    assert float((a - b).abs().max()) <= 1e-6 * float(a.abs().max())


def test_a_sequence_set_aside_and_resumed(folders, plains):
    """A copy of a sequence's pages, ring and memories goes on as the sequence itself does."""
    engine = model_for(folders, "A", "float32").engine
    tokens = tiny.prompt(140, tiny.ALL["A"]["vocab"], 17)
    ref = exact(plains, "A", tokens)
    a, b = engine.admit(2)
    engine.step([a], [tokens[:100]], [[]])
    engine.cache.copy_slot(a, b)
    one = torch.cat([engine.step([a], [[t]]).float().cpu() for t in tokens[100:]])
    two = engine.step([b], [tokens[100:]], [list(range(40))]).float().cpu()
    engine.release([a, b])
    check(one, ref[100:], "float32")
    check(two, ref[100:], "float32")


def test_constants_that_must_show(folders, plains, tmp_path):
    """Each constant and switch of the configuration moves the logits when it alone is changed (in the library and in the plain
    statement alike)."""
    from catena_models_b200.api import Model

    base = copy.deepcopy(tiny.TINY_A)
    tensors = tiny.make_tensors(base, 9)
    tokens = tiny.prompt(100, base["vocab"], 19)

    def ref_of(cfg):
        return plain.forward(tokens, {n: t.double() for n, t in tensors.items()}, cfg)[0]

    start = ref_of(base)
    for change in (lambda c: c["norm"].update(eps=0.05), lambda c: c["embedding"].update(scale=0.7),
                   lambda c: c["layers"][0]["mixer"].update(gate_cap=1.5), lambda c: c["layers"][1]["mixer"].update(softcap=1.0),
                   lambda c: c["layers"][1]["mixer"].pop("softcap"), lambda c: c["layers"][1]["mixer"]["rot"].pop("scaling"),
                   lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].update(original=400.0),
                   lambda c: c["layers"][1]["mixer"]["rot"].update(dims=10), lambda c: c["layers"][2]["mixer"]["mask"].update(size=21),
                   lambda c: c["layers"][2]["mixer"].update(scale=0.4), lambda c: c["layers"][2]["mixer"]["rot"].update(base=80.0),
                   lambda c: c["layers"][5]["mixer"]["rot"]["scaling"].update(factor=5.0)):
        cfg = copy.deepcopy(base)
        change(cfg)
        ref = ref_of(cfg)
        assert float((ref - start).abs().max() / start.abs().max()) > 1e-3
        folder = tiny.make_folder(tmp_path, "changed", config=cfg, tensors=tensors)
        check(run_alone(Model.load(folder, dtype="float32", max_tokens=512).engine, tokens, [60, 30]), ref, "float32")


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
            logits = run_alone(model_for(folders, "A", dtype, use_graphs=False).engine, seq, [len(p)]).double()
        for j, tok in enumerate(new):
            row = logits[len(p) - 1 + j]
            best = int(row.argmax())
            if tok != best:
                gap = float(row[best] - row[tok]) / float(row.abs().max())
                assert dtype == "bfloat16" and gap < 0.03, (tok, best, gap)


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
