"""The mechanisms that the Kofadra decoder added, each alone against the plain statement (plain_kofadra.py) or a float64
sum written here: the mask by chunks with a constant sink in every form of the attention kernels (whole prompts on the
CUDA cores, mma.sync and tcgen05; single tokens on the CUDA cores and mma.sync; portions on top of a paged cache in all
three forms), with a key that decides the row from the chunk's first position, and just outside it; the head norm over
padded heads; the gated delta rule as one kernel per token, row by row and in chunks; hyper-connected streams; the layer
norm; the router with a bias and a softmax over the chosen."""
import math
import types

import pytest
import torch

import plain_kofadra as plain
from test_kernels_gpu import DEV, _paged_cache, close, rnd

pytestmark = pytest.mark.gpu
F64 = torch.float64


@pytest.fixture(scope="module")
def K():
    from catena_models_b200 import kernels
    kernels.lib()
    return kernels


def masked_attention(q, k, v, window, scale, sink, first=0):
    """float64: rows `first`.. of the attention over the keys that row i sees: j <= i, and in i's chunk of -window rows
    (window < 0) or among the last `window` (window > 0); a score `sink` without a value joins the denominator (None: not)."""
    T, QH, HD = q.shape
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    hidden = j > i
    if window < 0:
        hidden |= torch.div(i, -window, rounding_mode="floor") != torch.div(j, -window, rounding_mode="floor")
    elif window > 0:
        hidden |= j + window <= i
    out = torch.zeros(T, QH, HD, dtype=F64)
    for h in range(QH):
        g = h // (QH // k.shape[1])
        s = ((q[:, h].double() @ k[:, g].double().T) * scale).masked_fill(hidden, -math.inf)
        if sink is not None:
            s = torch.cat([s, torch.full((T, 1), float(sink), dtype=F64)], 1)
        out[:, h] = torch.softmax(s, -1)[:, :T] @ v[:, g].double()
    return out[first:]


def _split(buf, QH, KVH, HD):
    return buf[:, :QH * HD], buf[:, QH * HD:(QH + KVH) * HD], buf[:, (QH + KVH) * HD:]


def _views(q, k, v, QH, KVH, HD):
    T = q.shape[0]
    return q.float().cpu().view(T, QH, HD), k.float().cpu().view(T, KVH, HD), v.float().cpu().view(T, KVH, HD)


def _prompt(K, impl, ctx, q, k, v, starts, B, longest, QH, KVH, HD, window, scale, sink):
    if impl == "tc":
        err = torch.zeros(1, dtype=torch.int32, device=DEV)
        K.attn_prefill_tc(ctx, q, k, v, None, starts, B, longest, QH, KVH, HD, window, scale, err=err, sink=sink)
        assert int(err) == 0
    else:
        fn = K.attn_prefill_mma if impl == "mma" else K.attn_prefill_simt
        fn(ctx, q, k, v, None, starts, B, longest, QH, KVH, HD, window, scale, sink=sink)


# ------------------------------------------------------------------------------------------ attention by chunks
@pytest.mark.parametrize("impl, dtype, QH, KVH, HD, T, chunk", [
    ("simt", torch.float32, 4, 2, 24, 150, 37), ("simt", torch.bfloat16, 3, 1, 40, 130, 64), ("simt", torch.float32, 2, 2, 16, 90, 1),
    ("mma", torch.bfloat16, 4, 2, 64, 300, 100), ("mma", torch.bfloat16, 2, 1, 112, 200, 7), ("mma", torch.bfloat16, 6, 6, 16, 140, 64),
    ("mma", torch.bfloat16, 2, 1, 96, 260, 65), ("tc", torch.bfloat16, 4, 2, 64, 900, 333), ("tc", torch.bfloat16, 2, 1, 128, 1000, 800),
    ("tc", torch.bfloat16, 2, 2, 64, 700, 130), ("tc", torch.bfloat16, 2, 1, 128, 600, 128), ("tc", torch.bfloat16, 2, 1, 64, 400, 5)])
def test_chunks_in_prompt_attention(K, impl, dtype, QH, KVH, HD, T, chunk):
    q, k, v = _split(rnd(T, (QH + 2 * KVH) * HD, dtype=dtype, seed=3), QH, KVH, HD)
    lens = [T - 70, 70]                                # two sequences side by side
    starts = torch.tensor([0, lens[0], T], dtype=torch.int32, device=DEV)
    sink = torch.zeros(QH, device=DEV)
    ctx = torch.empty(T, QH * HD, dtype=dtype, device=DEV)
    _prompt(K, impl, ctx, q, k, v, starts, 2, max(lens), QH, KVH, HD, -chunk, HD ** -0.5, sink)
    qv, kv, vv = _views(q, k, v, QH, KVH, HD)
    cut = ((0, lens[0]), (lens[0], T))
    ref = lambda w, s: torch.cat([masked_attention(qv[a:b], kv[a:b], vv[a:b], w, HD ** -0.5, s) for a, b in cut])
    close(ctx.view(T, QH, HD), ref(-chunk, 0.0), dtype)
    # a sliding window of that many positions, and a denominator without the sink, give other numbers on this input
    assert float((ref(-chunk, 0.0) - ref(-chunk, None)).abs().max()) > 0.05
    if chunk > 1:
        assert float((ref(-chunk, 0.0) - ref(chunk, 0.0)).abs().max()) > 0.05


@pytest.mark.parametrize("impl, dtype, HD, T", [("simt", torch.float32, 32, 400), ("mma", torch.bfloat16, 64, 400),
                                                ("tc", torch.bfloat16, 64, 900), ("tc", torch.bfloat16, 128, 900)])
@pytest.mark.parametrize("chunk, far", [(200, 200), (200, 399), (130, 130), (64, 191), (0, 0)])
def test_a_key_at_a_chunks_edge_in_prompts(K, impl, dtype, HD, T, chunk, far):
    """One key is made to stand out; exactly the queries from its position to the end of its chunk return its value."""
    QH, KVH = 2, 1
    q, k, v = _split(rnd(T, (QH + 2 * KVH) * HD, dtype=dtype, scale=0.3, seed=11), QH, KVH, HD)
    k[far] = 0
    k[far, 0] = 30.0
    q[:, 0] = 30.0                                     # every query of head 0 looks for it
    starts = torch.tensor([0, T], dtype=torch.int32, device=DEV)
    ctx = torch.empty(T, QH * HD, dtype=dtype, device=DEV)
    _prompt(K, impl, ctx, q, k, v, starts, 1, T, QH, KVH, HD, -chunk, HD ** -0.5, torch.zeros(QH, device=DEV))
    close(ctx.view(T, QH, HD), masked_attention(*_views(q, k, v, QH, KVH, HD), -chunk, HD ** -0.5, 0.0), dtype)
    hit = (ctx.view(T, QH, HD)[:, 0].float() - v[far].float()).abs().max(dim=-1).values < 0.05
    at = torch.arange(T, device=DEV)
    expect = at >= far
    if chunk:
        expect &= at < (far // chunk + 1) * chunk
    assert torch.equal(hit, expect)


@pytest.mark.parametrize("dtype, tensor_cores", [(torch.float32, False), (torch.bfloat16, False), (torch.bfloat16, True)])
@pytest.mark.parametrize("QH, KVH, HD, chunk", [(4, 2, 16, 1), (6, 3, 128, 90), (5, 5, 32, 70), (8, 2, 64, 320), (2, 1, 48, 64), (4, 1, 96, 300)])
def test_chunks_in_single_token_attention(K, dtype, tensor_cores, QH, KVH, HD, chunk):
    """Sequences that stand just before, on and behind a chunk's edge, in rings that have turned over."""
    K.set_decode_attention_tensor_cores(tensor_cores)
    K.set_decode_attention_target_blocks(3)            # blocks that walk several pieces
    try:
        ring = (chunk + 63) // 64 * 64
        lens, scale, n_chunks = [1, chunk, chunk + 1, 2 * chunk, 2 * chunk + 1, 3 * chunk - 1, 700], HD ** -0.5, -(-ring // 256)
        g = torch.Generator().manual_seed(HD + chunk)
        kv = [torch.randn(n, 2, KVH, HD, generator=g) for n in lens]
        pool, pages, ptab = _paged_cache(K, kv, KVH, HD, dtype, lens, ring)
        B = len(lens)
        q = rnd(B, QH * HD, dtype=dtype, scale=1.5, seed=7)
        pos = torch.tensor([n - 1 for n in lens], dtype=torch.int32, device=DEV)
        slots = torch.arange(1, B + 1, dtype=torch.int32, device=DEV)
        part_o, part_ml = K.attn_decode_scratch(B, QH, HD, n_chunks, DEV)
        ctx = torch.full((B, QH * HD), float("nan"), dtype=dtype, device=DEV)
        K.attn_decode(ctx, q, None, pos, slots, pool, pages, ptab, ring, -chunk, QH, KVH, HD, n_chunks, scale, part_o, part_ml,
                      sink=torch.zeros(QH, device=DEV))
        for b, n in enumerate(lens):
            kk, vv = kv[b][:, 0].to(dtype).float(), kv[b][:, 1].to(dtype).float()
            qq = torch.zeros(n, QH, HD)
            qq[-1] = q[b].float().cpu().view(QH, HD)
            close(ctx[b].view(QH, HD), masked_attention(qq, kk, vv, -chunk, scale, 0.0, first=n - 1)[0], dtype)
    finally:
        K.set_decode_attention_tensor_cores(True)
        K.set_decode_attention_target_blocks(0)


@pytest.mark.parametrize("dtype, tensor_cores", [(torch.float32, False), (torch.bfloat16, True)])
def test_a_key_at_a_chunks_edge_in_single_tokens(K, dtype, tensor_cores):
    """The key that stands out is found as the first of its chunk by the chunk's last token, and is gone one token later."""
    K.set_decode_attention_tensor_cores(tensor_cores)
    try:
        for chunk, far, n, seen in [(200, 200, 400, True), (200, 200, 401, False), (200, 199, 201, False), (64, 128, 192, True),
                                    (64, 128, 193, False), (90, 450, 451, True), (90, 449, 451, False), (300, 300, 600, True)]:
            ring = (chunk + 63) // 64 * 64
            kv = [torch.randn(n, 2, 1, 16, generator=torch.Generator().manual_seed(1)) * 0.1]
            kv[0][far, 0, 0] = 0.0
            kv[0][far, 0, 0, 0] = 40.0
            kv[0][far, 1, 0] = 7.0
            pool, pages, ptab = _paged_cache(K, kv, 1, 16, dtype, [n], ring)
            q = torch.zeros(1, 16, dtype=dtype, device=DEV)
            q[0, 0] = 40.0
            pos, slots = torch.tensor([n - 1], dtype=torch.int32, device=DEV), torch.tensor([1], dtype=torch.int32, device=DEV)
            part_o, part_ml = K.attn_decode_scratch(1, 1, 16, 2, DEV)
            ctx = torch.empty(1, 16, dtype=dtype, device=DEV)
            K.attn_decode(ctx, q, None, pos, slots, pool, pages, ptab, ring, -chunk, 1, 1, 16, 2, 0.25, part_o, part_ml,
                          sink=torch.zeros(1, device=DEV))
            if seen:
                assert torch.allclose(ctx.float().cpu(), torch.full((1, 16), 7.0), atol=5e-2), (chunk, far, n)
            else:
                assert float(ctx.float().abs().max()) < 1.0, (chunk, far, n)
    finally:
        K.set_decode_attention_tensor_cores(True)


@pytest.mark.parametrize("impl, dtype, QH, KVH, HD, chunk", [("simt", torch.float32, 4, 2, 24, 50), ("mma", torch.bfloat16, 4, 2, 64, 330),
                                                             ("mma", torch.bfloat16, 2, 1, 96, 90), ("tc", torch.bfloat16, 4, 1, 64, 600),
                                                             ("tc", torch.bfloat16, 2, 2, 128, 96), ("tc", torch.bfloat16, 2, 1, 64, 500)])
def test_chunks_in_portions_on_top_of_held_tokens(K, impl, dtype, QH, KVH, HD, chunk):
    past, new, scale = [0, 700, 65], [40, 130, 200], HD ** -0.5
    ring = (chunk + 63) // 64 * 64
    g = torch.Generator().manual_seed(5)
    seqs = [torch.randn(p + n, 3, max(QH, KVH), HD, generator=g) for p, n in zip(past, new)]
    kv = [s[:p, 1:, :KVH] for s, p in zip(seqs, past)]
    pool, pages, ptab = _paged_cache(K, kv, KVH, HD, dtype, past, ring)
    T = sum(new)
    buf = torch.cat([torch.cat([s[p:, 0, :QH].reshape(n, -1), s[p:, 1, :KVH].reshape(n, -1), s[p:, 2, :KVH].reshape(n, -1)], 1)
                     for s, p, n in zip(seqs, past, new)]).to(dtype).to(DEV)
    q, k, v = _split(buf, QH, KVH, HD)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=DEV)
    starts, pos0, slots, sink = i32([0, new[0], new[0] + new[1], T]), i32(past), i32([1, 2, 3]), torch.zeros(QH, device=DEV)
    ctx = torch.empty(T, QH * HD, dtype=dtype, device=DEV)
    if impl == "tc":
        err = torch.zeros(1, dtype=torch.int32, device=DEV)
        K.attn_append_tc(ctx, q, k, v, None, starts, pos0, slots, pool, pages, ptab, ring, 3, max(new), QH, KVH, HD, -chunk, scale,
                         err=err, sink=sink)
        assert int(err) == 0
    else:
        K.attn_append(ctx, q, k, v, None, starts, pos0, slots, pool, pages, ptab, ring, 3, max(new), QH, KVH, HD, -chunk, scale,
                      tensor_cores=impl == "mma", sink=sink)
    at = 0
    for s, p, n in zip(seqs, past, new):
        r = s.to(dtype).float()
        ref = masked_attention(r[:, 0, :QH], r[:, 1, :KVH], r[:, 2, :KVH], -chunk, scale, 0.0, first=p)
        close(ctx[at:at + n].view(n, QH, HD), ref, dtype)
        at += n


@pytest.mark.parametrize("dtype, tol", [(torch.float32, 2e-6), (torch.bfloat16, 8e-3)])
@pytest.mark.parametrize("T, real, HD", [(5, 12, 32), (5, 20, 24), (200, 12, 32), (200, 40, 64), (200, 16, 16)])
def test_head_norm_over_padded_heads(K, dtype, tol, T, real, HD):
    """Heads of `real` channels padded with zeros to HD: the mean of squares counts the real ones, the padding stays zero."""
    QH, KVH, eps = 3, 1, 1e-2
    g = torch.Generator().manual_seed(T + HD)
    x = torch.zeros(T, QH + 2 * KVH, HD)
    x[..., :real] = torch.randn(T, QH + 2 * KVH, real, generator=g) * 0.3
    wq, wk = (torch.nn.functional.pad(1 + 0.3 * torch.randn(real, generator=g), (0, HD - real)).to(DEV) for _ in range(2))
    qkv = x.view(T, -1).to(dtype).to(DEV)
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=DEV)
    K.qk_prepare(qkv, wq, wk, None, i32(list(range(T))), i32([0] * T), i32([0]), i32([T]), None, 0, None, 0, QH, KVH, HD, eps,
                 norm_dim=real)
    got = qkv.double().cpu().view(T, -1, HD)
    src = x.to(dtype).double()
    ref = torch.cat([plain.rms(src[:, :QH, :real], eps) * wq[:real].double().cpu(), plain.rms(src[:, QH:QH + 1, :real], eps) * wk[:real].double().cpu()], 1)
    assert float((got[:, :QH + KVH, :real] - ref).abs().max()) < tol * float(ref.abs().max())
    assert float(got[:, :QH + KVH, real:].abs().max() if real < HD else 0.0) == 0.0
    assert torch.equal(got[:, QH + KVH:], src[:, QH + KVH:])               # values are left as they are


# ------------------------------------------------------------------------------------------ gated delta rule
def _batch(lengths, starts, slots, kind):
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=DEV)
    tok_seq, tok_pos, seq_start = [], [], [0]
    for b, (n, p) in enumerate(zip(lengths, starts)):
        tok_seq += [b] * n
        tok_pos += list(range(p, p + n))
        seq_start.append(seq_start[-1] + n)
    return types.SimpleNamespace(tok_seq=i32(tok_seq), tok_pos=i32(tok_pos), seq_start=i32(seq_start), seq_pos0=i32(starts),
                                 seq_slot=i32(slots), B=len(lengths), T=sum(lengths), max_len=max(lengths), kind=kind, shared={},
                                 partial_sums_ok=False)


def _delta_part(W, H, G, D, DV, taps, eps, dtype, seed):
    """(part bound on the device, its tensors in float64, runtime)."""
    from catena_models_b200.engine.runtime import Runtime
    from catena_models_b200.parts import build_part

    part = build_part("mixer", "delta_rule", prefix="m.", hidden=W, heads=H, kv_heads=G, dim=D, value_dim=DV, taps=taps, eps=eps,
                      out_dtype="float32")
    g = torch.Generator().manual_seed(seed)
    P = {}
    for spec in part.all_tensor_specs():
        n = torch.randn(tuple(spec.shape), generator=g)
        tail = spec.name.split(".")[-1]
        t = {"conv": 0.6 * n, "A_log": 1.5 * n - 1.0, "dt_bias": n, "norm": 1 + 0.2 * n}.get(tail, n / spec.shape[-1] ** 0.5)
        P[spec.name] = t.to(torch.bfloat16)
    rt = Runtime(dtype, DEV)
    matrix = {s.name for s in part.all_tensor_specs() if s.role == "matrix"}
    part.bind_all({k: v.to(DEV).to(dtype if k in matrix else torch.float32) for k, v in P.items()}, rt)
    return part, {k: v.double() for k, v in P.items()}, rt


@pytest.mark.parametrize("dtype, tol", [(torch.float32, 2e-5), (torch.bfloat16, 3e-2)])
@pytest.mark.parametrize("W, H, G, D, DV, taps", [
    (32, 4, 2, 16, 24, 4), (24, 1, 1, 8, 8, 1), (40, 3, 3, 7, 9, 2), (64, 4, 1, 64, 128, 3), (48, 2, 1, 128, 64, 4), (32, 2, 2, 4, 36, 5),
    (40, 2, 1, 20, 132, 4), (32, 1, 1, 150, 40, 3), (32, 2, 1, 96, 200, 16), (32, 2, 1, 64, 64, 4), (40, 2, 2, 128, 128, 2)])
def test_delta_rule_whole_portions_single_tokens_and_slots(W, H, G, D, DV, taps, dtype, tol):
    """Three sequences of unequal length, whole, in portions, two tokens at a time and token by token, on slots that were
    used before; head sizes with and without the one-kernel step and the chunked form."""
    from catena_models_b200 import kernels
    from catena_models_b200.parts.recurrent import DeltaRule

    eps = 1e-5
    part, P, rt = _delta_part(W, H, G, D, DV, taps, eps, dtype, seed=W + D)
    m = dict(heads=H, kv_heads=G, dim=D, vdim=DV)
    lengths = [75, 1, 130]
    g = torch.Generator().manual_seed(3)
    xs = [torch.randn(n, W, generator=g).to(dtype) for n in lengths]
    want = [plain.delta_mixer(x.double(), P, "m.", m, eps) for x in xs]
    scale = max(float(w.abs().max()) for w in want)
    (n,) = part.state_spec().shape
    state = types.SimpleNamespace(tensor=torch.full((6, n), float("nan"), device=DEV))
    keep = DeltaRule.CHUNKED_MIN_ROWS
    try:
        for cuts, slots, least in (([1000] * 3, [0, 1, 2], 1), ([1000] * 3, [2, 0, 5], 1 << 30), ([7, 1, 65], [4, 2, 0], 20),
                                   ([2, 1, 2], [1, 0, 3], 48), ([50, 1, 64], [5, 4, 1], 1), ([1, 1, 1], [3, 5, 2], 48)):
            DeltaRule.CHUNKED_MIN_ROWS = least
            kernels.zero_slots(state.tensor.view(1, 6, -1), slots)
            at = [0, 0, 0]
            while any(a < L for a, L in zip(at, lengths)):
                live = [i for i in range(3) if at[i] < lengths[i]]
                take = [min(cuts[i], lengths[i] - at[i]) for i in live]
                kind = "prefill" if all(at[i] == 0 for i in live) else ("decode" if all(t == 1 for t in take) else "append")
                batch = _batch(take, [at[i] for i in live], [slots[i] for i in live], kind)
                y = part.forward(rt, batch, torch.cat([xs[i][at[i]:at[i] + t] for i, t in zip(live, take)]).to(DEV), state)
                row = 0
                for i, t in zip(live, take):
                    got, ref = y[row:row + t].double().cpu(), want[i][at[i]:at[i] + t]
                    assert float((got - ref).abs().max()) < tol * scale, (cuts, i, at[i])
                    at[i] += t
                    row += t
    finally:
        DeltaRule.CHUNKED_MIN_ROWS = keep


@pytest.mark.parametrize("form", ["step", "rows", "chunks"])
def test_delta_rule_finds_what_was_written_long_ago_and_corrects_what_is_written_twice(form):
    """With a decay that keeps everything, one key is written once, then hundreds of orthogonal ones; asking for it returns
    its value.  Written again with another value, it returns that one (a plain sum of outer products would return both)."""
    from catena_models_b200 import kernels

    H = G = 1
    D, DV, T, taps = 32, 16, 300, 1
    eye = torch.eye(D)
    k, q, v = torch.zeros(T, D), torch.zeros(T, D), torch.zeros(T, DV)
    for t in range(T):
        k[t] = eye[1 + t % (D - 1)]
        v[t] = 0.5 + 0.001 * t
    k[5], v[5] = eye[0], 3.0
    k[150], v[150] = eye[0], -2.0
    q[149], q[299] = eye[0], eye[0]
    big = 40.0                                         # silu(big x) of a unit vector is that vector, times big
    proj = torch.cat([q * big, k * big, v, torch.ones(T, DV)], 1).to(DEV)
    dev = lambda *s: torch.ones(*s, device=DEV)
    state = torch.zeros(1, kernels.delta_state_floats(H, G, D, DV, taps), device=DEV)
    out = torch.empty(T, DV, device=DEV)
    # beta = sigmoid(50) = 1; rate 1 with softplus(-100) = 0: the decay is one
    gates = torch.cat([torch.full((T, 1), 50.0), torch.full((T, 1), -100.0)], 1).to(DEV)
    args = (dev(2 * D + DV, taps), dev(H), torch.zeros(H, device=DEV), dev(H * DV), state)
    tail = (H, G, D, DV, 1.0, 1e-6, 1e-6)
    if form == "step":
        for t in range(T):
            kernels.delta_rule(out[t:t + 1], proj[t:t + 1], *args, _batch([1], [t], [0], "decode"), *tail,
                               x=dev(1, 4), w_gates=torch.tensor([[12.5] * 4, [-25.0] * 4], device=DEV))
    else:
        scratch = dev(kernels.delta_chunk_floats(1, T, H, D, DV)) if form == "chunks" else None
        kernels.delta_rule(out, proj, *args, _batch([T], [0], [0], "prefill"), *tail, gates=gates, chunk_scratch=scratch)
    S = state[0, :D * DV].view(D, DV).cpu()
    silu = lambda x: float(plain.silu(torch.tensor(x, dtype=F64)))
    assert torch.allclose(S[0], torch.full((DV,), silu(-2.0)), atol=1e-5)
    # the unit norm hides the size, so the sign tells which value came back
    assert bool((out[149] > 0).all()) and bool((out[299] < 0).all())
    for i in range(1, D):
        last = max(t for t in range(T) if float(k[t, i]) == 1.0)
        assert torch.allclose(S[i], torch.full((DV,), silu(0.5 + 0.001 * last)), atol=1e-5)


# ------------------------------------------------------------------------------------------ streams and norms
@pytest.mark.parametrize("dtype, tol", [(torch.float32, 3e-6), (torch.bfloat16, 6e-3)])
@pytest.mark.parametrize("S, W", [(1, 52), (2, 256), (3, 37), (4, 1024), (5, 8), (8, 132)])
def test_hyper_connected_streams(K, dtype, tol, S, W):
    """Opening, reading alone, and the write behind a sublayer together with the next read; terms in float and in the
    activation dtype, and a routed feed-forward's pieces with an index and weights."""
    rows, eps = 9, 1e-3
    g = torch.Generator().manual_seed(S + W)
    r = lambda *s: torch.randn(*s, generator=g)
    a, put, mix, w = r(S), r(S), r(S, S), 1 + 0.2 * r(W)
    dev = lambda t: t.to(DEV).float().contiguous()
    e = r(rows, W) + 0.7                                # a mean that the norm has to take off
    x = torch.empty(rows, S, W, device=DEV)
    n = torch.empty(rows, W, dtype=dtype, device=DEV)
    norm = lambda X: plain.layer_norm(plain.stream_read(X, a.double()), w.double(), eps)
    near = lambda got, ref, t=tol: float((got.double().cpu() - ref).abs().max()) < t * max(1.0, float(ref.abs().max()))
    K.hyper_connect(dev(e), n_out=n, read=dev(a), w=dev(w), eps=eps, out=x)
    X = torch.stack([e.double()] * S)
    assert torch.equal(x.cpu(), e[:, None].expand(rows, S, W)) and near(n, norm(X))
    X = r(S, rows, W).double().float()
    x = dev(X.permute(1, 0, 2))
    before = x.clone()
    n = torch.empty(rows, W, dtype=dtype, device=DEV)
    K.hyper_connect(x, n_out=n, read=dev(a), w=dev(w), eps=eps)
    assert torch.equal(x, before) and near(n, norm(X.double()))
    y1, y2 = r(rows, W), r(rows, W).to(dtype)
    pieces, index, wts = r(3 * rows, W), torch.randperm(3 * rows, generator=g)[:2 * rows].int(), torch.rand(2 * rows, generator=g)
    index[3] = -1                                       # no piece here
    y = y1.double() + 0.5 * y2.double()
    for i in range(2 * rows):
        if int(index[i]) >= 0:
            y[i // 2] += wts[i].double() * pieces[int(index[i])].double()
    terms = K.Terms([(dev(y1), 1.0, 1), (y2.to(DEV), 0.5, 1), (dev(pieces), 1.0, 2, index.to(DEV), wts.to(DEV))])
    ref = plain.stream_write(X.double(), mix.double(), put.double(), y)
    n = torch.empty(rows, W, dtype=dtype, device=DEV)
    K.hyper_connect(x, terms, dev(mix), dev(put), n_out=n, read=dev(a), w=dev(w), eps=eps)
    assert near(x, ref.permute(1, 0, 2), 3e-6) and near(n, norm(ref))
    if S > 1:                                           # the mix is read [from, to]
        assert not near(x, plain.stream_write(X.double(), mix.T.double(), put.double(), y).permute(1, 0, 2), 1e-2)
    x = before.clone()
    K.hyper_connect(x, terms, dev(mix), dev(put))       # the last write of a stack: no reader
    assert near(x, ref.permute(1, 0, 2), 3e-6)


@pytest.mark.parametrize("dtype, tol", [(torch.float32, 3e-6), (torch.bfloat16, 6e-3)])
@pytest.mark.parametrize("W", [52, 256, 1000])
def test_layer_norm_alone_and_behind_a_residual_sum(K, dtype, tol, W):
    rows, eps = 7, 1e-3
    g = torch.Generator().manual_seed(W)
    x, w, y = torch.randn(rows, W, generator=g) + 2.0, 1 + 0.2 * torch.randn(W, generator=g), torch.randn(rows, W, generator=g)
    n = torch.empty(rows, W, dtype=dtype, device=DEV)
    K.norm_f32in(n, x.to(DEV), w.to(DEV), eps, layer=True)
    ref = plain.layer_norm(x.double(), w.double(), eps)
    assert float((n.double().cpu() - ref).abs().max()) < tol * float(ref.abs().max())
    h = x.to(DEV)
    n = torch.empty(rows, W, dtype=dtype, device=DEV)
    K.residual_add_norm(h, K.Terms([(y.to(DEV), 0.5, 1)]), n, w.to(DEV), eps, layer=True)
    total = x.double() + 0.5 * y.double()
    ref = plain.layer_norm(total, w.double(), eps)
    assert float((h.double().cpu() - total).abs().max()) < 1e-5
    assert float((n.double().cpu() - ref).abs().max()) < tol * float(ref.abs().max())


# ------------------------------------------------------------------------------------------ router
@pytest.mark.parametrize("rows", [1, 9, 64, 65, 300])
@pytest.mark.parametrize("E, top", [(1, 1), (8, 3), (5, 5), (160, 6)])
def test_router_with_a_bias_and_a_softmax_over_the_chosen(K, rows, E, top):
    W = 40
    g = torch.Generator().manual_seed(rows + E)
    h, router, bias = torch.randn(rows, W, generator=g), torch.randn(E, W, generator=g) * 0.4, 2.0 * torch.randn(E, generator=g)
    ids = torch.empty(rows * top, dtype=torch.int32, device=DEV)
    wts = torch.empty(rows * top, dtype=torch.float32, device=DEV)
    tiles = K.moe_max_tiles(rows * top, E)
    perm = torch.empty(tiles * K.MOE_TILE_SIMT, dtype=torch.int32, device=DEV)
    dest = torch.empty(rows * top, dtype=torch.int32, device=DEV)
    work = torch.empty(K.moe_work_size(rows * top, E), dtype=torch.int32, device=DEV)
    K.moe_route(ids, wts, perm, dest, work, h.to(DEV), router.to(DEV), None, top, gate="softmax_chosen", bias=bias.to(DEV))
    P = {"x.router": router.double(), "x.router.b": bias.double()}
    want_ids, want_w = plain.route(h.double(), P, "x.", dict(experts=E, top=top))
    assert torch.equal(ids.view(rows, top).cpu().long(), want_ids)
    assert float((wts.view(rows, top).cpu().double() - want_w).abs().max()) < 1e-5
    pairs = dest.cpu().tolist()
    assert len(set(pairs)) == rows * top and [int(perm[d]) for d in pairs] == list(range(rows * top))
    if E == 8 and rows == 300:                          # the bias moves the choice, and the weights are not the softmax over all
        bare, _ = plain.route(h.double(), {**P, "x.router.b": 0 * bias.double()}, "x.", dict(experts=E, top=top))
        assert not torch.equal(bare, want_ids)
        full = torch.softmax(h.double() @ router.double().T + bias.double(), -1).gather(1, want_ids)
        assert float((full - want_w).abs().max()) > 0.05


@pytest.mark.parametrize("dtype, tensor_cores, tol", [("float32", True, 2e-5), ("bfloat16", True, 2e-2), ("bfloat16", False, 2e-2)])
@pytest.mark.parametrize("rows", [7, 300])
def test_routed_feed_forward(K, dtype, tensor_cores, tol, rows):
    from catena_models_b200.engine.runtime import Runtime
    from catena_models_b200.parts import build_part

    W, F, E, top = 64, 48, 6, 3
    f = dict(kind="moe", expert=dict(ff=F), router=dict(experts=E, top=top))
    g = torch.Generator().manual_seed(12)
    n = lambda *s: (torch.randn(*s, generator=g) / s[-1] ** 0.5).to(torch.bfloat16)
    P = {"m.router": n(E, W) * 4, "m.router.b": torch.randn(E, generator=g).to(torch.bfloat16)}
    for e in range(E):
        P.update({f"m.e{e}.gate": n(F, W) * 2, f"m.e{e}.up": n(F, W) * 2, f"m.e{e}.down": n(W, F)})
    rt = Runtime(getattr(torch, dtype), DEV)
    rt.grouped_tensor_cores = tensor_cores
    part = build_part("feed_forward", "routed_swiglu", prefix="m.", hidden=W, intermediate=F, experts=E, top=top,
                      gate="softmax_chosen", weight_on="output", bias_name="router.b")
    part.bind_all({k: v.to(DEV).to(getattr(torch, dtype)) if v.dim() == 2 else v.to(DEV) for k, v in P.items()}, rt)
    x = torch.randn(rows, W, generator=g).to(torch.bfloat16)
    batch = types.SimpleNamespace(kind="prefill", tok_seq=torch.zeros(rows, dtype=torch.int32, device=DEV), shared={}, partial_sums_ok=False)
    total = torch.zeros(rows, W, dtype=torch.float32, device=DEV)
    K.residual_add_norm(total, part.forward(rt, batch, x.to(DEV).to(getattr(torch, dtype))))
    ref, _ = plain.moe_ff(x.double(), {k: v.double() for k, v in P.items()}, "m.", f)
    assert float((total.double().cpu() - ref).abs().max()) < tol * float(ref.abs().max())
