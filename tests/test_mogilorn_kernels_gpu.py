"""The mechanisms that the Mogilorn decoder added, each alone against the plain statement (plain_mogilorn.py) or a float64 sum
written here: the output gate per channel and the compact rows in every form of the attention kernels (with capped scores),
biases, head norms, rotations, mixed values and the cache write as one kernel, the norm on what is added to the stream, the
tanh-gelu in the products' epilogues, the matrix memory, and the latent attention with a window over a ring and a sink, with a
key that decides the row just inside and just outside the window, in prompts, in portions and in single tokens."""
import math
import types

import pytest
import torch

import plain_mogilorn as plain
from test_kernels_gpu import DEV, _paged_cache, close, rnd
from test_maferax_kernels_gpu import _batch, _close

pytestmark = pytest.mark.gpu
F64 = torch.float64


@pytest.fixture(scope="module")
def K():
    from catena_models_b200 import kernels
    kernels.lib()
    return kernels


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


# ------------------------------------------------------------------------------------------ attention's output
def attention_rows(q, k, v, window, scale, cap, sink, gate, DV, channels, first=0):
    """float64: rows `first`.. of a causal attention with capped scores, an optional window and sink, its first DV value channels
    times sigmoid of gate [T, H] or [T, H, DV]."""
    T, QH, HD = q.shape
    back = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    hidden = (back < 0) | ((back >= window) if window else torch.zeros_like(back, dtype=torch.bool))
    out = torch.zeros(T, QH, DV, dtype=F64)
    for h in range(QH):
        g = h // (QH // k.shape[1])
        s = plain.soft_cap((q[:, h].double() @ k[:, g].double().T) * scale, cap).masked_fill(hidden, -math.inf)
        if sink is not None:
            s = torch.cat([s, torch.full((T, 1), float(sink[h]), dtype=F64)], 1)
        out[:, h] = torch.softmax(s, -1)[:, :T] @ v[:, g, :DV].double()
    gate = gate.double() if channels else gate.double()[:, :, None]
    return (out * torch.sigmoid(gate))[first:]


def _gates(T, QH, DV, channels, dtype, seed):
    """Gate logits inside wider rows whose pitch is a multiple of 8."""
    n = QH * (DV if channels else 1)
    wide = rnd(T, -(-n // 8) * 8 + 8, dtype=dtype, scale=1.5, seed=seed)
    return wide[:, :n], wide[:, :n].float().cpu().view((T, QH, DV) if channels else (T, QH))


FORMS = [("simt", torch.float32, 4, 2, 32, 32), ("simt", torch.float32, 3, 1, 48, 21), ("simt", torch.bfloat16, 2, 2, 160, 100),
         ("mma", torch.bfloat16, 4, 2, 64, 64), ("mma", torch.bfloat16, 2, 1, 80, 50), ("mma", torch.bfloat16, 3, 3, 16, 6),
         ("tc", torch.bfloat16, 4, 2, 64, 64), ("tc", torch.bfloat16, 4, 1, 64, 40), ("tc", torch.bfloat16, 2, 1, 128, 128),
         ("tc", torch.bfloat16, 2, 2, 128, 72)]


@pytest.mark.parametrize("channels", [True, False])
@pytest.mark.parametrize("impl, dtype, QH, KVH, HD, DV", FORMS)
def test_gates_per_channel_and_compact_rows_in_prompts(K, impl, dtype, QH, KVH, HD, DV, channels):
    T, cap, window = 500, 6.0, 0 if DV == HD else 170
    buf = rnd(T, (QH + 2 * KVH) * HD, dtype=dtype, seed=3)
    q, k, v = buf[:, :QH * HD], buf[:, QH * HD:(QH + KVH) * HD], buf[:, (QH + KVH) * HD:]
    gate, gref = _gates(T, QH, DV, channels, dtype, 5)
    sink = rnd(QH, seed=9) if window else None
    lens = [T - 190, 190]
    starts = i32([0, lens[0], T])
    ctx = torch.full((T, QH * DV), float("nan"), dtype=dtype, device=DEV)
    extra = dict(sink=sink, softcap=cap, value_dim=DV, gate_channels=channels)
    if impl == "tc":
        err = torch.zeros(1, dtype=torch.int32, device=DEV)
        K.attn_prefill_tc(ctx, q, k, v, gate, starts, 2, max(lens), QH, KVH, HD, window, 0.3, err=err, **extra)
        assert int(err) == 0
    else:
        fn = K.attn_prefill_mma if impl == "mma" else K.attn_prefill_simt
        fn(ctx, q, k, v, gate, starts, 2, max(lens), QH, KVH, HD, window, 0.3, **extra)
    f = lambda x, n: x.float().cpu().view(T, n, HD)
    for a, b in ((0, lens[0]), (lens[0], T)):
        ref = attention_rows(f(q, QH)[a:b], f(k, KVH)[a:b], f(v, KVH)[a:b], window, 0.3, cap, None if sink is None else sink.cpu(),
                             gref[a:b], DV, channels)
        close(ctx[a:b].view(-1, QH, DV), ref, dtype)


@pytest.mark.parametrize("channels", [True, False])
@pytest.mark.parametrize("dtype, tensor_cores, QH, KVH, HD, DV", [
    (torch.float32, False, 4, 2, 32, 20), (torch.bfloat16, False, 4, 2, 64, 64), (torch.bfloat16, True, 8, 2, 64, 48),
    (torch.bfloat16, True, 3, 1, 128, 128), (torch.float32, False, 2, 1, 160, 130)])
def test_gates_per_channel_and_compact_rows_in_single_tokens(K, dtype, tensor_cores, QH, KVH, HD, DV, channels):
    K.set_decode_attention_tensor_cores(tensor_cores)
    try:
        lens, scale, cap = [1, 64, 65, 700], 0.2, 5.0
        g = torch.Generator().manual_seed(HD)
        kv = [torch.randn(n, 2, KVH, HD, generator=g) for n in lens]
        pool, pages, ptab = _paged_cache(K, kv, KVH, HD, dtype, lens, 0)
        B = len(lens)
        q = rnd(B, QH * HD, dtype=dtype, scale=1.5, seed=7)
        gate, gref = _gates(B, QH, DV, channels, dtype, 6)
        part_o, part_ml = K.attn_decode_scratch(B, QH, HD, 3, DEV)
        ctx = torch.full((B, QH * DV), float("nan"), dtype=dtype, device=DEV)
        K.attn_decode(ctx, q, gate, i32([n - 1 for n in lens]), torch.arange(1, B + 1, dtype=torch.int32, device=DEV), pool, pages,
                      ptab, 0, 0, QH, KVH, HD, 3, scale, part_o, part_ml, softcap=cap, value_dim=DV, gate_channels=channels)
        for b, n in enumerate(lens):
            kk, vv = kv[b][:, 0].to(dtype).float(), kv[b][:, 1].to(dtype).float()
            qq = torch.zeros(n, QH, HD)
            qq[-1] = q[b].float().cpu().view(QH, HD)
            gg = torch.zeros(n, *gref.shape[1:])
            gg[-1] = gref[b]
            close(ctx[b].view(QH, DV), attention_rows(qq, kk, vv, 0, scale, cap, None, gg, DV, channels, first=n - 1)[0], dtype)
    finally:
        K.set_decode_attention_tensor_cores(True)


@pytest.mark.parametrize("impl, dtype, QH, KVH, HD, DV", FORMS)
def test_gates_per_channel_in_portions_on_top_of_held_tokens(K, impl, dtype, QH, KVH, HD, DV):
    past, new, scale, cap = [0, 300, 65], [40, 130, 100], 0.2, 7.0
    g = torch.Generator().manual_seed(5)
    seqs = [torch.randn(p + n, 3, max(QH, KVH), HD, generator=g) for p, n in zip(past, new)]
    pool, pages, ptab = _paged_cache(K, [s[:p, 1:, :KVH] for s, p in zip(seqs, past)], KVH, HD, dtype, past, 0)
    T = sum(new)
    buf = torch.cat([torch.cat([s[p:, 0, :QH].reshape(n, -1), s[p:, 1, :KVH].reshape(n, -1), s[p:, 2, :KVH].reshape(n, -1)], 1)
                     for s, p, n in zip(seqs, past, new)]).to(dtype).to(DEV)
    q, k, v = buf[:, :QH * HD], buf[:, QH * HD:(QH + KVH) * HD], buf[:, (QH + KVH) * HD:]
    gate, gref = _gates(T, QH, DV, True, dtype, 8)
    starts, pos0, slots = i32([0, new[0], new[0] + new[1], T]), i32(past), i32([1, 2, 3])
    ctx = torch.full((T, QH * DV), float("nan"), dtype=dtype, device=DEV)
    args = (ctx, q, k, v, gate, starts, pos0, slots, pool, pages, ptab, 0, 3, max(new), QH, KVH, HD, 0, scale)
    extra = dict(softcap=cap, value_dim=DV, gate_channels=True)
    if impl == "tc":
        err = torch.zeros(1, dtype=torch.int32, device=DEV)
        K.attn_append_tc(*args, err=err, **extra)
        assert int(err) == 0
    else:
        K.attn_append(*args, tensor_cores=impl == "mma", **extra)
    at = 0
    for s, p, n in zip(seqs, past, new):
        r = s.to(dtype).float()
        gg = torch.zeros(p + n, QH, DV)
        gg[p:] = gref[at:at + n]
        close(ctx[at:at + n].view(n, QH, DV),
              attention_rows(r[:, 0, :QH], r[:, 1, :KVH], r[:, 2, :KVH], 0, scale, cap, None, gg, DV, True, first=p), dtype)
        at += n


def test_rows_that_a_form_cannot_store_are_refused(K):
    buf = rnd(40, 3 * 64, dtype=torch.bfloat16)
    q, k, v = buf[:, :64], buf[:, 64:128], buf[:, 128:]
    ctx = torch.empty(40, 64, dtype=torch.bfloat16, device=DEV)
    for fn, dv in ((K.attn_prefill_mma, 33), (K.attn_prefill_tc, 36), (K.attn_prefill_simt, 65)):
        with pytest.raises(K.KernelError):
            fn(ctx, q, k, v, None, i32([0, 40]), 1, 40, 1, 1, 64, 0, 0.1, value_dim=dv)
    gate = rnd(40, 67, dtype=torch.bfloat16)
    for fn in (K.attn_prefill_mma, K.attn_prefill_tc):
        with pytest.raises(K.KernelError):
            fn(ctx, q, k, v, gate[:, 1:65], i32([0, 40]), 1, 40, 1, 1, 64, 0, 0.1, gate_channels=True)


# ------------------------------------------------------------------------------------------ heads in front of the attention
def _turned(x, pos, rate, pairs, interleaved):
    """x [T, heads, HD]: the leading `pairs` pairs turned by pos * rate."""
    HD, out = x.shape[-1], x.clone()
    for i in range(pairs):
        lo, hi = (2 * i, 2 * i + 1) if interleaved else (i, i + HD // 2)
        a = (pos.float() * rate[i]).double()[:, None]                  # the angle is a float32 product
        out[..., lo] = x[..., lo] * torch.cos(a) - x[..., hi] * torch.sin(a)
        out[..., hi] = x[..., hi] * torch.cos(a) + x[..., lo] * torch.sin(a)
    return out


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("QH, KVH, HD, dim, dv, pairs, interleaved, normed, biased, first, ring", [
    (4, 2, 16, 16, 16, 8, True, True, True, None, 0), (3, 1, 32, 20, 30, 7, True, True, True, (3, 10, 16), 64),
    (8, 2, 64, 64, 64, 32, True, True, True, (2, 64, 64), 0), (2, 2, 48, 48, 40, 12, True, True, False, (4, 20, 32), 128),
    (5, 5, 112, 112, 112, 56, False, True, True, None, 64), (4, 1, 128, 128, 128, 64, False, False, True, (2, 64, 64), 0),
    (2, 1, 256, 256, 200, 0, False, True, False, (1, 200, 208), 0), (6, 3, 80, 72, 80, 3, True, False, True, None, 0)])
def test_head_prepare(K, dtype, QH, KVH, HD, dim, dv, pairs, interleaved, normed, biased, first, ring):
    """Rows of three sequences (one of which stands on held tokens) and rows of padding; heads padded with zeros; values mixed
    with values that come in another number of heads with another padding."""
    lengths, starts, slots = [150, 3, 70], [0, 7, 60], [2, 0, 3]
    batch = _batch(lengths, starts, slots)
    T, pad = batch.T, 5
    batch.tok_seq = torch.cat([batch.tok_seq, i32([-1] * pad)])
    batch.tok_pos = torch.cat([batch.tok_pos, i32([0] * pad)])
    g = torch.Generator().manual_seed(HD + dim)
    live = lambda heads, n: torch.nn.functional.pad(torch.randn(T + pad, heads, n, generator=g), (0, HD - n)).reshape(T + pad, -1)
    width = (QH + 2 * KVH) * HD
    rows = torch.cat([live(QH, dim), live(KVH, dim), live(KVH, dv), torch.randn(T + pad, 8, generator=g)], 1).to(dtype)
    padded = lambda heads, n: torch.nn.functional.pad(torch.randn(heads, n, generator=g), (0, HD - n)).reshape(-1)
    bias = torch.cat([padded(QH, dim), padded(KVH, dim), padded(KVH, dv)]) if biased else None
    wq, wk = ((1 + 0.3 * padded(1, dim)) * (torch.arange(HD) < dim) for _ in range(2)) if normed else (None, None)
    rate = torch.rand(pairs, generator=g) if pairs else None
    mix, lam = None, torch.tensor([0.3], device=DEV)
    if first is not None:
        h1, dv1, hd1 = first
        assert h1 * dv1 == KVH * dv
        src = torch.randn(T + pad, h1 * hd1 + 8, generator=g).to(dtype)
        mix = (src.to(DEV)[:, :h1 * hd1], dv1, hd1, lam)
    pages = 12
    pool = torch.full((2, pages, KVH, 64, HD), 77.0, dtype=dtype, device=DEV)
    ptab = torch.randperm(pages, generator=g).view(4, 3).to(DEV, torch.int32)
    dev = lambda t: None if t is None else t.to(DEV)
    out = rows.to(DEV)
    K.head_prepare(out, batch, QH, KVH, HD, bias=dev(bias), wq=dev(wq), wk=dev(wk), norm_dim=dim, eps=1e-5, rate=dev(rate),
                   interleaved=interleaved, value_dim=dv, mix=mix, kv=(pool, pages, ptab, ring))
    assert torch.equal(out[T:].cpu(), rows[T:]) and torch.equal(out[:, width:].cpu(), rows[:, width:])       # padding, and what is behind v
    x = rows[:T, :width].double() + (0 if bias is None else bias.double())
    q, k, v = x[:, :QH * HD].view(T, QH, HD), x[:, QH * HD:(QH + KVH) * HD].view(T, KVH, HD), x[:, (QH + KVH) * HD:].view(T, KVH, HD)
    pos = batch.tok_pos[:T].cpu()
    if normed:
        q, k = (u / torch.sqrt((u * u).sum(-1, keepdim=True) / dim + 1e-5) * w.double() for u, w in ((q, wq), (k, wk)))
    if pairs:
        q, k = _turned(q, pos, rate, pairs, interleaved), _turned(k, pos, rate, pairs, interleaved)
    if first is not None:
        other = src[:T, :h1 * hd1].double().view(T, h1, hd1)[:, :, :dv1].reshape(T, KVH, dv)
        v = v.clone()
        v[:, :, :dv] = plain.mix_values(v[:, :, :dv], other, float(lam))
    want = torch.cat([u.reshape(T, -1) for u in (q, k, v)], 1)
    close(out[:T, :width], want, dtype)
    # the cache holds the rows exactly as they were written back; a ring keeps the last `ring` positions of each sequence
    at = 0
    for n, p, s in zip(lengths, starts, slots):
        for j in range(n):
            if ring and p + j + ring < p + n:
                continue
            e = (p + j) % ring if ring else p + j
            page = int(ptab[s, e // 64])
            got = out[at + j, QH * HD:width].view(2, KVH, HD)
            if j % 17 == 0 or j == n - 1:
                assert torch.equal(pool[:, page, :, e % 64], got)
        at += n
    # without a cache the rows are the same
    again = rows.to(DEV)
    K.head_prepare(again, batch, QH, KVH, HD, bias=dev(bias), wq=dev(wq), wk=dev(wk), norm_dim=dim, eps=1e-5, rate=dev(rate),
                   interleaved=interleaved, value_dim=dv, mix=mix)
    assert torch.equal(again, out)


# ------------------------------------------------------------------------------------------ the norm on what is added
@pytest.mark.parametrize("dtype, tol", [(torch.float32, 3e-6), (torch.bfloat16, 6e-3)])
@pytest.mark.parametrize("W", [52, 77, 256, 2048, 3000, 8192, 9000])
def test_norm_on_what_is_added(K, dtype, tol, W):
    g = torch.Generator().manual_seed(W)
    rows = 19
    h, a, b, bias = torch.randn(rows, W, generator=g) * 2, torch.randn(rows, W, generator=g), torch.randn(rows, W, generator=g), torch.randn(W, generator=g)
    pieces, wts = torch.randn(rows * 3, W, generator=g), torch.rand(rows * 3, generator=g)
    w, w_next = torch.randn(W, generator=g) * 0.5, 1 + 0.3 * torch.randn(W, generator=g)
    act = b.to(dtype)
    for many in (False, True):
        total = a.double() + 0.5 * act.double() + bias.double()
        terms = [(a.to(DEV), 1.0, 1), (act.to(DEV), 0.5, 1), (bias.to(DEV), 1.0, 0)]
        if many:                                   # a term of several weighted pieces a row
            total = total + (wts.double()[:, None] * pieces.double()).view(rows, 3, W).sum(1)
            terms.append((pieces.to(DEV), 1.0, 3, None, wts.to(DEV)))
        want = h.double() + plain.one_plus(total, w.double(), 1e-5)
        w_dev = (1 + w).to(DEV)
        hd, n_out = h.to(DEV).clone(), torch.empty(rows, W, dtype=dtype, device=DEV)
        K.outnorm_residual(hd, K.Terms(terms), w_dev, 1e-5, n_out=n_out)
        _close(hd, want, 3e-6)
        _close(n_out, want, tol)
        hd = h.to(DEV).clone()
        K.outnorm_residual(hd, K.Terms(terms), w_dev, 1e-5, n_out=n_out, w_next=w_next.to(DEV), eps_next=1e-3)
        _close(hd, want, 3e-6)
        _close(n_out, plain.rms(want, 1e-3) * w_next.double(), tol)
        hd = h.to(DEV).clone()
        K.outnorm_residual(hd, K.Terms(terms), w_dev, 1e-5)
        _close(hd, want, 3e-6)


def test_a_bias_in_the_other_residual_sums(K):
    g = torch.Generator().manual_seed(2)
    h, a, bias, w = torch.randn(9, 40, generator=g), torch.randn(9, 40, generator=g), torch.randn(40, generator=g), torch.rand(40, generator=g)
    terms = K.Terms([(a.to(DEV), 1.0, 1), (bias.to(DEV), 2.0, 0)])
    want = h.double() + a.double() + 2 * bias.double()
    hd = h.to(DEV).clone()
    K.residual_add_norm(hd, terms)
    _close(hd, want, 3e-6)
    hd = h.to(DEV).clone()
    K.postnorm_residual(hd, terms, 1.0, w.to(DEV), 1e-5)
    _close(hd, plain.rms(want, 1e-5) * w.double(), 3e-6)
    with pytest.raises(K.KernelError):
        K.residual_add_norm(hd, K.Terms([(a.to(DEV), 1.0, 0)]))


# ------------------------------------------------------------------------------------------ plain gelu in the products
@pytest.mark.parametrize("rows", [1, 8, 9, 16, 17, 40, 64, 65, 128, 129, 300, 700])
@pytest.mark.parametrize("N, Kd", [(320, 256), (1000, 2048), (56, 40)])
def test_gelu_in_the_products_epilogues(K, rows, N, Kd):
    from catena_models_b200.engine.runtime import Runtime

    rt = Runtime(torch.bfloat16, DEV)
    x, w = rnd(rows, Kd, dtype=torch.bfloat16, seed=1), rnd(N, Kd, dtype=torch.bfloat16, scale=3.0 * Kd ** -0.5, seed=2)
    ref = plain.gelu_tanh(x.double().cpu() @ w.double().cpu().T)
    got = rt.linear_gelu(x, w)
    rt.check_errors()
    assert float(((got.double().cpu() - ref).abs() / (ref.abs() + 0.05)).max()) < 1e-2
    rt.tensor_core_prompts, rt._in_prompt = False, True              # the CUDA-core product and the activation behind it
    _close(rt.linear_gelu(x, w), ref, 1e-2)
    rt32 = Runtime(torch.float32, DEV)
    _close(rt32.linear_gelu(x.float(), w.float()), ref, 1e-5)


@pytest.mark.parametrize("block_n", [128, 192, 256])
def test_gelu_in_every_tile_width(K, block_n):
    x, w = rnd(333, 264, dtype=torch.bfloat16, seed=1), rnd(520, 264, dtype=torch.bfloat16, scale=0.2, seed=2)
    err = torch.zeros(1, dtype=torch.int32, device=DEV)
    y = torch.empty(333, 520, dtype=torch.bfloat16, device=DEV)
    K.gemm_tc(y, x, w, swiglu=K.GATE_GELU, err=err, block_n=block_n)
    assert int(err) == 0
    _close(y, plain.gelu_tanh(x.double().cpu() @ w.double().cpu().T), 6e-3)


def test_gelu_far_from_zero(K):
    z = torch.tensor([-300.0, -60.0, -9.0, -4.0, -1.0, -1e-3, 0.0, 1e-3, 1.0, 4.0, 9.0, 60.0, 300.0])
    x = torch.zeros(16, 64)
    x[:13, 0] = z
    w = torch.zeros(64, 64)
    w[:, 0] = 1.0
    y = torch.empty(16, 64, dtype=torch.bfloat16, device=DEV)
    K.gemm_skinny(y, x.to(DEV, torch.bfloat16), w.to(DEV, torch.bfloat16), swiglu=K.GATE_GELU)
    ref = plain.gelu_tanh(z.to(torch.bfloat16).double())
    assert bool(torch.isfinite(y).all()) and float((y[:13, 5].double().cpu() - ref).abs().max() / 300) < 3e-3
    assert float((y[:8, 5].double().cpu() - ref[:8]).abs().max()) < 2e-3
    a = z.to(DEV).clone()
    K.act_inplace(a, "gelu_tanh")
    _close(a, plain.gelu_tanh(z.double()), 1e-6)


# ------------------------------------------------------------------------------------------ matrix memory
@pytest.mark.parametrize("H, D, DV", [(1, 8, 8), (3, 16, 24), (2, 7, 9), (4, 64, 32)])
def test_matrix_memory_scan_with_gates_of_any_strength(K, H, D, DV):
    """The scan against the plain recurrence from a state of zeros whose maximum starts at zero: gates that keep everything, gates
    that forget within a token, input gates far below and far above the maximum; whole, in portions, on a slot used before."""
    from catena_models_b200.parts import build_part

    g = torch.Generator().manual_seed(H * D)
    T = 130
    q, k, v, gate = (torch.randn(T, H, n, generator=g) for n in (D, D, DV, DV))
    i = torch.randn(T, H, generator=g) * 4.0
    f = torch.nn.functional.logsigmoid(torch.randn(T, H, generator=g) * 4.0)
    i[40] = 12.0                                          # one token that outweighs what was there
    i[:3] = -9.0                                          # the first tokens stay below the starting maximum
    o, _ = plain.mlstm_scan(q.double() * D ** -0.5, k.double(), v.double(), i.double(), f.double())
    norm_w = 1 + 0.3 * torch.randn(H * DV, generator=g)
    want = plain.rms(o, 1e-5).reshape(T, -1) * norm_w.double() * torch.sigmoid(gate.double().reshape(T, -1))
    part = build_part("mixer", "matrix_memory", prefix="m.", hidden=8, heads=H, dim=D, value_dim=DV, gate_cap=1.0, eps=1e-5)
    state = torch.zeros(3, part.state_spec().shape[0], device=DEV)
    gates = torch.cat([i, f], 1).to(DEV)
    rows = [u.reshape(T, -1).to(DEV) for u in (q, k, v, gate)]
    for cuts in ([T], [1] * T, [2, 63, 64, 1]):
        state[1] = 0
        out, at = torch.empty(T, H * DV, device=DEV), 0
        for n in cuts:
            s = slice(at, at + n)
            K.matrix_scan("memory", out[s], *(u[s] for u in rows), gates[s].contiguous(), None, norm_w.to(DEV), state, 0, i32([0, n]),
                          i32([1]), 1, H, D, DV, D ** -0.5, 1e-5)
            at += n
        _close(out, want, 2e-5)
    assert float(state[0].abs().max()) == 0.0 and float(state[2].abs().max()) == 0.0


# ------------------------------------------------------------------------------------------ latents: window, ring, sink
def _latent_part(W, m, dtype, window, seed):
    from catena_models_b200.engine.runtime import Runtime
    from catena_models_b200.parts import build_part

    g = torch.Generator().manual_seed(seed)
    H, D, R, DV, KR = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    mat = lambda o, n, s=1.0: torch.randn(o, n, generator=g) * s / n ** 0.5
    P = {"m.q": mat(H * (D + R), W, 2.0), "m.dkv": mat(KR + R, W), "m.uk": mat(H * D, KR), "m.uv": mat(H * DV, KR), "m.g": mat(H * DV, W),
         "m.o": mat(W, H * DV), "m.dkv.norm": 1 + 0.3 * torch.randn(KR, generator=g), "m.sink": torch.randn(H, generator=g) * 1.5}
    if dtype == torch.bfloat16:
        P = {n: t.to(torch.bfloat16).float() for n, t in P.items()}
    position = build_part("position", "paired_rotary", dims=m["rot"]["dims"], theta=m["rot"]["base"]) if R else build_part("position", "none")
    rt = Runtime(dtype, DEV)
    part = build_part("mixer", "latent_attention", prefix="m.", hidden=W, heads=H, dim=D, rot_dim=R, value_dim=DV, kv_rank=KR, q_rank=None,
                      position=position, scale=m["scale"], eps=1e-5, gate_channels=True, window=window, sink_name="sink",
                      out_dtype="float32")
    part.bind_all({k: v.to(DEV, dtype if v.dim() == 2 else torch.float32) for k, v in P.items()}, rt)
    return rt, part, {k: v.double() for k, v in P.items()}


@pytest.mark.parametrize("dtype, tol", [(torch.float32, 2e-5), (torch.bfloat16, 2.5e-2)])
@pytest.mark.parametrize("H, D, R, DV, KR, W, window", [
    (3, 16, 8, 24, 40, 64, 20), (1, 12, 6, 20, 21, 36, 1), (2, 8, 2, 8, 16, 32, 64), (4, 32, 16, 64, 64, 128, 65), (5, 8, 4, 8, 136, 40, 0),
    (2, 40, 24, 72, 32, 64, 100), (17, 8, 0, 8, 8, 24, 33)])
def test_latent_attention_with_a_window_and_a_sink(K, dtype, tol, H, D, R, DV, KR, W, window):
    """The mixer over pages in any order: three unequal sequences as whole prompts, in portions down to one token, and on slots
    whose ring has been used before; every row against the plain statement."""
    m = dict(heads=H, dim=D, rot_dim=R, vdim=DV, kv_rank=KR, scale=0.35, rot=dict(dims=R, base=60.0) if R else None, mask=dict(size=window))
    rt, part, P = _latent_part(W, m, dtype, window, 6)
    g = torch.Generator().manual_seed(7)
    lengths = [230, 3, 90]
    xs = [torch.randn(n, W, generator=g) for n in lengths]
    if dtype == torch.bfloat16:
        xs = [x.to(torch.bfloat16).float() for x in xs]
    refs = [plain.latent_attention(x.double(), P, "m.", m, 1e-5) for x in xs]
    spec = part.state_spec()
    assert (spec.planes, spec.head_dim, spec.ring) == (1, -(-(KR + R) // 8) * 8, -(-window // 64) * 64)
    per = spec.ring // 64 or 4
    pool = torch.full((1, 6 * per + 1, 1, 64, spec.head_dim), float("nan"), dtype=dtype, device=DEV)
    ptab = torch.randperm(6 * per, generator=g).view(6, per).to(DEV, torch.int32)
    state = types.SimpleNamespace(pool=pool, ptab=ptab, spec=spec)

    def run(cuts, slots, whole):
        outs, at = [torch.empty(n, W) for n in lengths], [0, 0, 0]
        while any(at[i] < lengths[i] for i in range(3)):
            rows, lens, starts, sl, who = [], [], [], [], []
            for i in range(3):
                n = min(cuts[i], lengths[i] - at[i])
                if n > 0:
                    rows.append(xs[i][at[i]:at[i] + n])
                    lens.append(n); starts.append(at[i]); sl.append(slots[i]); who.append(i)
                    at[i] += n
            kind = "prefill" if whole and not any(starts) else None
            b = _batch(lens, starts, sl, kind=kind)
            b.append, b.prefill = b.kind == "append", b.kind == "prefill"
            y = part.forward(rt, b, torch.cat(rows).to(DEV, dtype), state).float().cpu()
            rt.check_errors()
            o = 0
            for i, n, s in zip(who, lens, starts):
                outs[i][s:s + n] = y[o:o + n]
                o += n
        return outs

    for cuts, slots, whole in (([1000] * 3, [0, 1, 2], True), ([1000] * 3, [0, 1, 2], False), ([7, 1, 33], [4, 2, 0], False),
                               ([64, 2, 1], [1, 5, 3], False), ([200, 1, 60], [2, 0, 4], True), ([2, 2, 2], [3, 1, 5], False),
                               ([1, 1, 1], [0, 2, 4], True)):
        for got, ref in zip(run(cuts, slots, whole), refs):
            _close(got, ref, tol)


@pytest.mark.parametrize("H, D, R, DV, KR, W, window", [
    (4, 32, 16, 64, 64, 128, 333), (2, 64, 32, 48, 128, 96, 900), (3, 24, 8, 128, 72, 64, 70), (2, 16, 8, 24, 40, 64, 0)])
def test_latent_attention_windows_in_long_prompts(K, H, D, R, DV, KR, W, window):
    """Whole bfloat16 prompts long enough for the tensor-core attention kernels: keys and values expanded per head, under the
    window, with the sink and the gate per channel, then single tokens that read the ring which that step left."""
    m = dict(heads=H, dim=D, rot_dim=R, vdim=DV, kv_rank=KR, scale=0.3, rot=dict(dims=R, base=60.0), mask=dict(size=window))
    rt, part, P = _latent_part(W, m, torch.bfloat16, window, 11)
    g = torch.Generator().manual_seed(12)
    lengths, tail = [1100, 65, 300], 3
    xs = [torch.randn(n + tail, W, generator=g).to(torch.bfloat16).float() for n in lengths]
    refs = [plain.latent_attention(x.double(), P, "m.", m, 1e-5) for x in xs]
    spec = part.state_spec()
    per = spec.ring // 64 or 18
    pool = torch.full((1, 3 * per, 1, 64, spec.head_dim), float("nan"), dtype=torch.bfloat16, device=DEV)
    state = types.SimpleNamespace(pool=pool, ptab=torch.randperm(3 * per, generator=g).view(3, per).to(DEV, torch.int32), spec=spec)
    b = _batch(lengths, [0, 0, 0], [0, 1, 2], kind="prefill")
    b.append, b.prefill = False, True
    y = part.forward(rt, b, torch.cat([x[:n] for x, n in zip(xs, lengths)]).to(DEV, torch.bfloat16), state).float().cpu()
    for got, ref, n in zip(torch.split(y, lengths), refs, lengths):
        _close(got, ref[:n], 2.5e-2)
    for t in range(tail):
        b = _batch([1, 1, 1], [n + t for n in lengths], [0, 1, 2])
        b.append, b.prefill = False, False
        y = part.forward(rt, b, torch.stack([x[n + t] for x, n in zip(xs, lengths)]).to(DEV, torch.bfloat16), state).float().cpu()
        for i, n in enumerate(lengths):
            _close(y[i], refs[i][n + t], 3e-2)
    rt.check_errors()


def _latent_sum(qa, keys, row, window, sink, KR, scale):
    """float64: heads' sums over the latents that position `row` sees; qa [H, E], keys [n, E], sink [H]."""
    first = max(0, row - window + 1) if window else 0
    s = torch.einsum("he,ne->hn", qa.double(), keys[first:row + 1].double()) * scale
    return plain.sink_softmax(s[:, None], sink.double())[:, 0] @ keys[first:row + 1, :KR].double()


@pytest.mark.parametrize("form", ["portion", "single", "tensor cores"])
@pytest.mark.parametrize("window", [1, 20, 64, 65, 200])
def test_a_latent_key_at_a_windows_edge(K, form, window):
    """One key stands out, and the sum is its row exactly as long as the row sees it: as the row itself, just behind the window's
    edge, one position outside it, at page borders and after the ring has turned over; the ring holds other sequences' leavings."""
    H, R, KR = 3, 8, 40
    E, EC, ring = KR + R, 48, -(-window // 64) * 64
    g = torch.Generator().manual_seed(8)
    base = torch.randn(760, E, generator=g) * 0.3
    ptab = torch.full((2, ring // 64), -1, dtype=torch.int32, device=DEV)
    order = torch.randperm(ring // 64 + 3, generator=g)[:ring // 64].tolist()
    ptab[1] = torch.tensor(order, dtype=torch.int32)
    sink = torch.tensor([-1.0, 0.5, 3.0])
    mma = form == "tensor cores"
    dtype = torch.bfloat16 if mma else torch.float32
    for row in (699, 128, 64, 63, window, window - 1, 300):
        for key in {row, max(0, row - window + 1), max(0, row - window), max(0, row - 1)}:
            direction = torch.randn(E, generator=g)
            keys = base.clone()
            keys[key] += 8.0 * direction / direction.norm()
            qa = torch.randn(1, H, E, generator=g) * 0.3
            qa[0, 1] += 8.0 * direction / direction.norm()
            if mma:
                keys, qa = keys.to(dtype).float(), qa.to(dtype).float()
            first = row if form != "portion" else max(0, row - 2)
            held = first + 1 if form != "portion" else first                # positions in the ring when the attention runs
            pool = torch.full((1, ring // 64 + 3, 1, 64, EC), 50.0, device=DEV, dtype=dtype)
            for p in range(max(0, held - ring), held):
                e = p % ring
                pool[0, order[e // 64], 0, e % 64, :E] = keys[p].to(DEV, dtype)
                pool[0, order[e // 64], 0, e % 64, E:] = 0
            if form == "portion":
                b = _batch([row + 2 - first], [first], [1])
                rows = torch.randn(b.T, H, E, generator=g) * 0.3
                rows[row - first] = qa[0]
                entries = torch.zeros(b.T, EC, device=DEV)
                entries[:, :E] = keys[first:row + 2].to(DEV)
            else:
                b, rows, entries = _batch([1], [row], [1], kind="decode"), qa, None
            ref = _latent_sum(qa[0], keys, row, window, sink, KR, 1.0)
            loud = float((ref[1] - keys[key, :KR].double()).abs().max()) < 0.5
            assert loud == (row - window < key <= row)
            for keys_hint in ((0, 1024) if form != "portion" else (0,)):
                splits, chunk, parts = 1, 0, None
                if keys_hint:
                    splits, chunk = K.latent_attn_splits(1, H, min(keys_hint, window) + 32, heads_per_block=16 if mma else 32)
                    parts = torch.full((H * splits * (2 + KR),), float("nan"), device=DEV)
                out = torch.full((b.T, H * KR), float("nan"), device=DEV)
                K.latent_attn(out, rows.reshape(b.T, H * E).to(DEV), None, pool, ptab, b, H, R, KR, 1.0, splits=splits, chunk=chunk,
                              parts=parts, tensor_cores=mma, window=window, ring=ring, sink=sink.to(DEV), entries=entries)
                _close(out[row - first].view(H, KR), ref, 6e-3 if mma else 2e-5)


@pytest.mark.parametrize("HD", [64, 128])
@pytest.mark.parametrize("far, window", [(0, 0), (3, 0), (511, 0), (512, 0)])
def test_a_far_key_under_a_gate_per_channel(K, HD, far, window):
    """A key hundreds of positions back decides the rows that look for it, capped scores or not."""
    QH, KVH, T = 2, 1, 900
    buf = rnd(T, (QH + 2 * KVH) * HD, dtype=torch.bfloat16, scale=0.3, seed=11)
    q, k, v = buf[:, :QH * HD], buf[:, QH * HD:(QH + KVH) * HD], buf[:, (QH + KVH) * HD:]
    k[far] = 0
    k[far, 0] = 30.0
    q[:, 0] = 30.0
    gate, gref = _gates(T, QH, HD, True, torch.bfloat16, 4)
    for cap in (0.0, 60.0):
        ctx = torch.empty(T, QH * HD, dtype=torch.bfloat16, device=DEV)
        err = torch.zeros(1, dtype=torch.int32, device=DEV)
        K.attn_prefill_tc(ctx, q, k, v, gate, i32([0, T]), 1, T, QH, KVH, HD, window, HD ** -0.5, err=err, softcap=cap, gate_channels=True)
        assert int(err) == 0
        f = lambda x, n: x.float().cpu().view(T, n, HD)
        close(ctx.view(T, QH, HD), attention_rows(f(q, QH), f(k, KVH), f(v, KVH), window, HD ** -0.5, cap, None, gref, HD, True), torch.bfloat16)
        hit = ctx.view(T, QH, HD)[far:, 0].float().cpu()
        assert float((hit - v[far].float().cpu() * torch.sigmoid(gref[far:, 0])).abs().max()) < 0.05
