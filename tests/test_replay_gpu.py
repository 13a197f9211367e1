"""bin/trace_run as a user drives it: a subprocess fed JSON lines on standard input.  The same
requests whole, with the last 32 tokens one by one, in unequal batches one after another
(so slots and pages are used again), and with their prompts cut into two steps (the second on
top of what the first left, while another request starts beside it), in 32-bit and in bfloat16,
against the plain model."""
import json
import os
import subprocess

import numpy as np
import pytest
import torch

import plain_lfm3
import tiny

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def replay(folder, dtype, steps, out_dir, max_tokens):
    lines = "".join(json.dumps(s) + "\n" for s in steps)
    run = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out",
                          str(out_dir), "--max-tokens", str(max_tokens)], input=lines, capture_output=True,
                         text=True, timeout=900)
    assert run.returncode == 0, run.stderr[-2000:]
    assert [l for l in run.stdout.splitlines() if l.startswith("done")] == [f"done {s['step']}" for s in steps]
    return run


def read(out_dir, step, vocab):
    return torch.from_numpy(np.fromfile(os.path.join(str(out_dir), f"{step}.f32"), dtype="<f4").reshape(-1, vocab).copy())


def rel(got, ref):
    return float((got.double() - ref.double()).abs().max() / ref.double().abs().max())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B"])
def test_replay_four_ways(tmp_path, name, dtype):
    folder = tiny.make_folder(tmp_path, name, seed=7)
    cfg, tensors = plain_lfm3.load_folder(folder)
    V = cfg["vocab_size"]
    lens = {"a": 40, "b": 97, "c": 33, "d": 130, "e": 35}
    reqs = {k: tiny.random_prompt(n, V, seed=ord(k)) for k, n in lens.items()}
    steps, expect, way_of = [], {}, {}          # expect[step] = list of (request, positions)
    n = 0
    way = "whole"

    def add(entries, end=()):
        nonlocal n
        steps.append({"step": n, "entries": entries, "end": list(end)})
        wanted = [(e["id"].split(":")[0], e["_pos"]) for e in entries if e["want"]]
        for e in entries:
            del e["_pos"]
        if wanted:
            expect[n] = wanted
            way_of[n] = way
        n += 1

    # 1) each request alone and whole, every position wanted
    for k, toks in reqs.items():
        add([{"id": f"{k}:w", "tokens": toks, "want": list(range(len(toks))), "_pos": list(range(len(toks)))}], end=[f"{k}:w"])
    # 2) the last 32 tokens one by one after a prompt step of the rest
    way = "tail"
    for k, toks in reqs.items():
        head = len(toks) - 32
        add([{"id": f"{k}:t", "tokens": toks[:head], "want": [head - 1], "_pos": [head - 1]}])
        for t in range(head, len(toks)):
            add([{"id": f"{k}:t", "tokens": [toks[t]], "want": [0], "_pos": [t]}], end=[f"{k}:t"] if t == len(toks) - 1 else [])
    # 3) batches of unequal lengths: prompts of different sizes, the shorter requests end earlier;
    #    a step with nothing wanted in between; the next batch starts on the freed slots
    way = "batch"
    for batch, prompt_lens in ((["a", "b", "c"], [8, 60, 1]), (["d", "e", "a"], [100, 3, 39])):
        ids = [f"{k}:b" for k in batch]
        add([{"id": i, "tokens": reqs[k][:p], "want": [0, p - 1] if p > 1 else [0], "_pos": [0, p - 1] if p > 1 else [0]}
             for i, k, p in zip(ids, batch, prompt_lens)])
        pos = dict(zip(batch, prompt_lens))
        live = list(batch)
        quiet = True
        while live:
            entries, ending = [], []
            for k in live:
                want = [] if (quiet and k == live[0]) else [0]
                entries.append({"id": f"{k}:b", "tokens": [reqs[k][pos[k]]], "want": want, "_pos": [pos[k]] if want else []})
                pos[k] += 1
                if pos[k] == len(reqs[k]):
                    ending.append(k)
            quiet = False
            add(entries, end=[f"{k}:b" for k in ending])
            live = [k for k in live if k not in ending]
    # 4) prompts in two chunks: every request brings its second chunk on top of its first, in one batch
    #    with unequal cuts, while a request that has not started yet joins with its whole prompt
    way = "chunks"
    cuts = {"a": 13, "b": 64, "c": 1, "d": 100}
    add([{"id": f"{k}:c", "tokens": reqs[k][:c], "want": [c - 1], "_pos": [c - 1]} for k, c in cuts.items()])
    entries = [{"id": f"{k}:c", "tokens": reqs[k][c:], "want": list(range(len(reqs[k]) - c)),
                "_pos": list(range(c, len(reqs[k])))} for k, c in cuts.items()]
    entries.append({"id": "e:c", "tokens": reqs["e"], "want": list(range(len(reqs["e"]))), "_pos": list(range(len(reqs["e"])))})
    add(entries, end=[f"{k}:c" for k in reqs])
    out = tmp_path / "out"
    # peak: the chunked batch holds 40 + 97 + 33 + 130 + 35 tokens -> 64 + 128 + 64 + 192 + 64 = 512
    replay(folder, dtype, steps, out, max_tokens=512)
    exact = {k: plain_lfm3.forward(cfg, tensors, t) for k, t in reqs.items()}
    same = {k: plain_lfm3.forward(cfg, tensors, t, bf16=True) for k, t in reqs.items()} if dtype == "bfloat16" else None
    assert sorted(int(f[:-4]) for f in os.listdir(out)) == sorted(expect)
    # Gather the rows of each (request, way) over all its steps: the bfloat16 criterion compares
    # the engine's distance from the exact model with the distance of the plain model run with
    # the reference's bfloat16 rounding points, and both are maxima over the same set of rows.
    rows = {}
    for step, wanted in expect.items():
        got = read(out, step, V)
        assert got.shape[0] == sum(len(p) for _, p in wanted)
        off = 0
        for key, positions in wanted:
            rows.setdefault((key, way_of[step]), []).append((got[off:off + len(positions)], positions))
            off += len(positions)
    assert len(rows) == 20                                   # five requests, four ways
    for (k, way), parts in rows.items():
        got = torch.cat([g for g, _ in parts])
        pos = [p for _, ps in parts for p in ps]
        ref = exact[k][pos]
        if dtype == "float32":
            assert rel(got, ref) < 2e-5, (k, way)
        else:
            assert rel(got, ref) < 2.0 * rel(same[k][pos], ref), (k, way)


def test_replay_refuses_what_does_not_fit(tmp_path):
    folder = tiny.make_folder(tmp_path, "A", seed=7)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": [1] * 200, "want": [199]}], "end": []}]
    lines = "".join(json.dumps(s) + "\n" for s in steps)
    run = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", "float32", "--out",
                          str(tmp_path / "o"), "--max-tokens", "128"], input=lines, capture_output=True, text=True,
                         timeout=600)
    assert run.returncode != 0 and "page" in run.stderr


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["Q", "D"])
def test_replay_of_a_narasun_model(tmp_path, name, dtype):
    """The second architecture through the same program: a request whole, one with its last tokens one by one, and
    three unequal requests that start together (one of a single token) and decode together until each has ended."""
    import plain_narasun
    import tiny_narasun

    folder = tiny_narasun.make_folder(tmp_path, name, seed=3)
    cfg, tensors = tiny_narasun.load_plain(folder)
    V = cfg["vocab"]
    reqs = {k: tiny_narasun.prompt(n, V, seed=ord(k)) for k, n in {"a": 1, "b": 70, "c": 135, "d": 90}.items()}
    exact = {k: plain_narasun.forward(cfg, tensors, t) for k, t in reqs.items()}
    same = {k: plain_narasun.forward(cfg, tensors, t, bf16=True) for k, t in reqs.items()} if dtype == "bfloat16" else exact
    _replay_whole_tail_and_together(tmp_path, folder, V, reqs, exact, same, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B"])
def test_replay_of_a_fozedra_model(tmp_path, name, dtype):
    """The third architecture through the same program, on the same schedule."""
    import plain_fozedra
    import tiny_fozedra

    folder = tiny_fozedra.make_folder(tmp_path, name, seed=5)
    cfg, tensors = tiny_fozedra.load_plain(folder)
    V = cfg["vocab"]
    reqs = {k: tiny_fozedra.prompt(n, V, seed=ord(k)) for k, n in {"a": 1, "b": 70, "c": 135, "d": 90}.items()}
    exact = {k: plain_fozedra.forward(cfg, tensors, t) for k, t in reqs.items()}
    same = ({k: plain_fozedra.forward(cfg, tensors, t, rd=plain_fozedra.to_bf16) for k, t in reqs.items()}
            if dtype == "bfloat16" else exact)
    _replay_whole_tail_and_together(tmp_path, folder, V, reqs, exact, same, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "M"])
def test_replay_of_a_maferax_model(tmp_path, name, dtype):
    """The fourth architecture through the same program, on the same schedule (in bfloat16 the whole prompts take the
    expanded form of the latent attention and the single tokens its tensor-core form)."""
    import plain_maferax
    import tiny_maferax

    folder = tiny_maferax.make_folder(tmp_path, name, seed=6)
    cfg, tensors = tiny_maferax.load_plain(folder)
    V = cfg["vocab"]
    reqs = {k: tiny_maferax.prompt(n, V, seed=ord(k)) for k, n in {"a": 1, "b": 70, "c": 135, "d": 90}.items()}
    exact, same = {}, {}
    for k, t in reqs.items():
        if dtype == "bfloat16":
            # the exact model follows the experts that the rounded one chose: a close call is no error of the program
            ids = {}
            same[k] = plain_maferax.forward(t, tensors, cfg, rd=plain_maferax.to_bf16, ids_out=ids)[0]
            exact[k] = plain_maferax.forward(t, tensors, cfg, expert_ids=ids)[0]
        else:
            exact[k] = same[k] = plain_maferax.forward(t, tensors, cfg)[0]
    _replay_whole_tail_and_together(tmp_path, folder, V, reqs, exact, same, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "M"])
def test_replay_of_a_relilix_model(tmp_path, name, dtype):
    """The fifth architecture through the same program, on the same schedule (windows shorter than the prompts, rings
    that turn over while the requests decode together, a layer that reads another layer's latents)."""
    import plain_relilix
    import tiny_relilix

    folder = tiny_relilix.make_folder(tmp_path, name, seed=7)
    cfg, tensors = tiny_relilix.load_plain(folder)
    V = cfg["vocab"]
    reqs = {k: tiny_relilix.prompt(n, V, seed=ord(k)) for k, n in {"a": 1, "b": 70, "c": 135, "d": 90}.items()}
    if dtype == "bfloat16":
        # Behind a window of a few tokens one choice of experts that rounding turns colours every row that still sees the
        # token, so the bfloat16 replay is held against the library itself stepping the same schedule in this process
        # (its arithmetic is checked against the plain statement where the experts it chose can be watched).
        _replay_whole_tail_and_together(tmp_path, folder, V, reqs, None, None, dtype, against_library=True)
        return
    exact = {k: plain_relilix.forward(t, tensors, cfg)[0] for k, t in reqs.items()}
    _replay_whole_tail_and_together(tmp_path, folder, V, reqs, exact, exact, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "M"])
def test_replay_of_a_kofadra_model(tmp_path, name, dtype):
    """The sixth architecture through the same program, on the same schedule (chunks that end in prompts and in decoding,
    states of every pass of a loop); bfloat16 as for the fifth."""
    import plain_kofadra
    import tiny_kofadra

    folder = tiny_kofadra.make_folder(tmp_path, name, seed=7)
    cfg, tensors = tiny_kofadra.load_plain(folder)
    V = cfg["vocab"]
    reqs = {k: tiny_kofadra.prompt(n, V, seed=ord(k)) for k, n in {"a": 1, "b": 70, "c": 135, "d": 90}.items()}
    if dtype == "bfloat16":
        _replay_whole_tail_and_together(tmp_path, folder, V, reqs, None, None, dtype, against_library=True)
        return
    exact = {k: plain_kofadra.forward(t, tensors, cfg)[0] for k, t in reqs.items()}
    _replay_whole_tail_and_together(tmp_path, folder, V, reqs, exact, exact, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "M"])
def test_replay_of_a_mogilorn_model(tmp_path, name, dtype):
    """The seventh architecture through the same program, on the same schedule (windows whose edge passes over prompts and over
    decoded tokens, memories, mixed values); bfloat16 as for the fifth."""
    import plain_mogilorn
    import tiny_mogilorn

    folder = tiny_mogilorn.make_folder(tmp_path, name, seed=7)
    cfg, tensors = tiny_mogilorn.load_plain(folder)
    V = cfg["vocab"]
    reqs = {k: tiny_mogilorn.prompt(n, V, seed=ord(k)) for k, n in {"a": 1, "b": 70, "c": 135, "d": 90}.items()}
    if dtype == "bfloat16":
        _replay_whole_tail_and_together(tmp_path, folder, V, reqs, None, None, dtype, against_library=True)
        return
    exact = {k: plain_mogilorn.forward(t, tensors, cfg)[0] for k, t in reqs.items()}
    _replay_whole_tail_and_together(tmp_path, folder, V, reqs, exact, exact, dtype)


def _library_steps(folder, dtype, steps, max_tokens):
    """The same schedule through the library's engine in this process: {step: logits of its wanted places}."""
    from catena_models_b200.api import Model

    engine = Model.load(folder, dtype=dtype, max_tokens=max_tokens + 64 * 64).engine
    slots, out = {}, {}
    for rec in steps:
        for e in rec["entries"]:
            if e["id"] not in slots:
                (slots[e["id"]],) = engine.admit(1)
        logits = engine.step([slots[e["id"]] for e in rec["entries"]], [list(e["tokens"]) for e in rec["entries"]],
                             [list(e["want"]) for e in rec["entries"]])
        if logits.shape[0]:
            out[rec["step"]] = logits.float().cpu()
        for rid in rec["end"]:
            engine.release([slots.pop(rid)])
    engine.check_errors()
    return out


def _replay_whole_tail_and_together(tmp_path, folder, V, reqs, exact, same, dtype, against_library=False):
    """Requests a (1 token), b (70), c (135), d (90): c whole; d with its last 30 tokens one by one; a, b and c started
    together and decoded together until each has ended."""
    steps, expect = [], {}

    def add(entries, positions, end=()):
        steps.append({"step": len(steps), "entries": entries, "end": list(end)})
        if positions:
            expect[len(steps) - 1] = positions

    add([{"id": "w", "tokens": reqs["c"], "want": list(range(135))}], [("c", p) for p in range(135)], end=["w"])
    add([{"id": "t", "tokens": reqs["d"][:60], "want": [0, 59]}], [("d", 0), ("d", 59)])
    for p in range(60, 90):
        add([{"id": "t", "tokens": [reqs["d"][p]], "want": [0]}], [("d", p)], end=["t"] if p == 89 else [])
    heads = {"a": 1, "b": 40, "c": 100}
    add([{"id": k, "tokens": reqs[k][:n], "want": [n - 1]} for k, n in heads.items()], [(k, n - 1) for k, n in heads.items()],
        end=["a"])
    at = dict(heads)
    live = ["b", "c"]
    while live:
        entries = [{"id": k, "tokens": [reqs[k][at[k]]], "want": [0] if at[k] % 3 else []} for k in live]
        positions = [(k, at[k]) for k in live if at[k] % 3]
        for k in live:
            at[k] += 1
        done = [k for k in live if at[k] == len(reqs[k])]
        add(entries, positions, end=done)
        live = [k for k in live if k not in done]
    out = tmp_path / "o"
    replay(folder, dtype, steps, out, max_tokens=1 + 70 + 135)
    if against_library:
        mine = _library_steps(folder, dtype, steps, 1 + 70 + 135)
        assert sorted(mine) == sorted(expect)
        for step in expect:
            a, b = read(out, step, V), mine[step]
            assert a.shape == b.shape and float((a - b).abs().max()) <= 1e-6 * float(b.abs().max()), step
        return
    got, ref, yard = [], [], []
    for step, positions in expect.items():
        got.append(read(out, step, V))
        ref += [exact[k][p] for k, p in positions]
        yard += [same[k][p] for k, p in positions]
    got, ref, yard = torch.cat(got), torch.stack(ref), torch.stack(yard)
    errs = (got.double() - ref.double()).abs().amax(-1) / ref.double().abs().amax(-1)
    if dtype == "float32":
        assert float(errs.max()) < 3e-5
    else:
        base = (yard.double() - ref.double()).abs().amax(-1) / ref.double().abs().amax(-1)
        # Q routes one expert of three per token: a close call may fall the other way in bfloat16 (for single rows)
        assert float(errs.median()) < 2.0 * float(base.median()) + 0.004
        assert float((errs > 3.0 * float(torch.quantile(base, 0.9)) + 0.016).double().mean()) <= 0.15
