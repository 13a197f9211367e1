"""Plain statement of the Mogilorn decoder, one function per mechanism, in float64 on the CPU.

Nothing here is shared with the library: the tests compare the engine's kernels with these functions.  `P` is
{tensor name: float64 tensor}; `cfg` is the dict of config.json; h [T, W] are the rows of one sequence from position 0.

    one_plus(x, w)    x / sqrt(mean(x^2) + eps) * (1 + w)
    embedding         E[token] * s_e
    sublayer          x <- x + one_plus(f(x), w)                 (f reads the stream itself)
    output            one_plus(x, w_f) E^T

`rd` (default: nothing) is applied wherever an engine that keeps activations in bfloat16 would round: the rows that the
products read, the products' results, the cached rows.  With `to_bf16` the functions give the yardstick for what the
storage format alone costs.
"""
import math

import torch

F64 = torch.float64


def ident(x):
    return x


def to_bf16(x):
    return x.to(torch.bfloat16).to(x.dtype)


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def one_plus(x, w, eps):
    return rms(x, eps) * (1.0 + w)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rotation_rates(rot):
    """Angle per position of every pair; with `scaling` long wavelengths are stretched by `factor`, short ones kept, and
    the ones between the two borders blended by where their wavelength lies."""
    sc, out = rot.get("scaling"), []
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        if sc:
            wave = 2.0 * math.pi / f
            if wave > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            elif wave >= sc["original"] / sc["high"]:
                s = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
                f = (1.0 - s) * f / sc["factor"] + s * f
        out.append(f)
    return torch.tensor(out, dtype=F64)


def turn(x, rot):
    """x [T, heads, n] of positions 0 .. T - 1: channels (2i, 2i + 1) of the leading `dims` turned, the others kept."""
    if not rot:
        return x
    d, out = rot["dims"], x.clone()
    ang = (torch.arange(x.shape[0], dtype=F64)[:, None] * rotation_rates(rot)[None])[:, None, :]
    u, v = x[..., 0:d:2], x[..., 1:d:2]
    out[..., 0:d:2] = u * torch.cos(ang) - v * torch.sin(ang)
    out[..., 1:d:2] = v * torch.cos(ang) + u * torch.sin(ang)
    return out


def soft_cap(s, cap):
    return cap * torch.tanh(s / cap) if cap else s


def visible(T, size):
    """[T, T]: query i may look at key j; `size` > 0 keeps the last `size` positions, itself among them."""
    back = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (back >= 0) & (back < size) if size else back >= 0


def sink_softmax(s, sink=None):
    """Weights exp(s_j) / (sum_j exp(s_j) + exp(sink)) along the last axis; s [H, T, N] with -inf for hidden keys,
    sink [H] or None."""
    mx = s.max(-1, keepdim=True).values
    if sink is not None:
        mx = torch.maximum(mx, sink[:, None, None])
    e = torch.exp(s - mx)
    den = e.sum(-1, keepdim=True)
    if sink is not None:
        den = den + torch.exp(sink[:, None, None] - mx)
    return e / den


def mix_values(v, v_first, lam):
    return (1.0 - lam) * v + lam * v_first


def attention(h, P, p, m, eps, v_first=None, rd=ident):
    """(y, v): v [T, G * DV] are the layer's own values (before any mixing), v_first those of the first mixing layer."""
    T, H, G = h.shape[0], m["heads"], m.get("kv_heads", m["heads"])
    D, DV = m["dim"], m.get("vdim", m["dim"])
    proj = lambda s: h @ P[p + s].T + P[p + s + ".b"]
    q = rms(rd(proj("q")).view(T, H, D), eps) * P[p + "q.norm"]
    k = rms(rd(proj("k")).view(T, G, D), eps) * P[p + "k.norm"]
    q, k = rd(turn(q, m.get("rot"))), rd(turn(k, m.get("rot")))
    own = rd(proj("v"))
    v = own if v_first is None else rd(mix_values(own, v_first, P[p + "vmix"]))
    k, v = k.repeat_interleave(H // G, 1), v.view(T, G, DV).repeat_interleave(H // G, 1)
    s = soft_cap(torch.einsum("thd,nhd->htn", q, k) * m["scale"], m.get("softcap"))
    w = sink_softmax(s.masked_fill(~visible(T, 0)[None], float("-inf")))
    o = torch.einsum("htn,nhv->thv", w, v).reshape(T, H * DV)
    o = rd(o * torch.sigmoid(rd(h @ P[p + "g"].T)))
    return o @ P[p + "o"].T + P[p + "o.b"], own


def mlstm_scan(q, k, v, i, f, state=None):
    """q, k [T, H, D], v [T, H, DV], log gates i, f [T, H]; state (S [H, D, DV], n [H, D], m [H]) or None.
    Returns (o [T, H, DV], state)."""
    T, H, D = q.shape
    S, n, m = state or (torch.zeros(H, D, v.shape[2], dtype=F64), torch.zeros(H, D, dtype=F64), torch.zeros(H, dtype=F64))
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for t in range(T):
        new = torch.maximum(f[t] + m, i[t])
        a, b = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        S = a[:, None, None] * S + b[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = a[:, None] * n + b[:, None] * k[t]
        m = new
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out[t] = torch.einsum("hdv,hd->hv", S, q[t]) / den[:, None]
    return out, (S, n, m)


def capped(z, cap):
    return cap * torch.tanh(z / cap)


def mlstm(h, P, p, m, eps, rd=ident):
    T, H, D, DV = h.shape[0], m["heads"], m["dim"], m.get("vdim", m["dim"])
    q, k, v = rd(h @ P[p + "q"].T).view(T, H, D) * D ** -0.5, rd(h @ P[p + "k"].T).view(T, H, D), rd(h @ P[p + "v"].T).view(T, H, DV)
    i = capped(h @ P[p + "i"].T + P[p + "i.b"], m["gate_cap"])
    f = torch.nn.functional.logsigmoid(capped(h @ P[p + "f"].T + P[p + "f.b"], m["gate_cap"]))
    o, _ = mlstm_scan(q, k, v, i, f)
    o = rms(o, eps).reshape(T, H * DV) * P[p + "norm"] * torch.sigmoid(rd(h @ P[p + "g"].T))
    return rd(o) @ P[p + "o"].T


def latent_attention(h, P, p, m, eps, rd=ident):
    T, H, D, R = h.shape[0], m["heads"], m["dim"], m["rot_dim"]
    DV, KR = m.get("vdim", D), m["kv_rank"]
    q = rd(h @ P[p + "q"].T).view(T, H, D + R)
    low = rd(h @ P[p + "dkv"].T)
    c = rd(rms(low[:, :KR], eps) * P[p + "dkv.norm"])
    r = rd(turn(low[:, None, KR:], m.get("rot")))[:, 0]
    q_turn = turn(q[..., D:], m.get("rot"))
    k, v = (c @ P[p + "uk"].T).view(T, H, D), (c @ P[p + "uv"].T).view(T, H, DV)
    s = (torch.einsum("thd,nhd->htn", q[..., :D], k) + torch.einsum("thr,nr->htn", q_turn, r)) * m["scale"]
    s = s.masked_fill(~visible(T, (m.get("mask") or {}).get("size", 0))[None], float("-inf"))
    o = torch.einsum("htn,nhv->thv", sink_softmax(s, P[p + "sink"]), v).reshape(T, H * DV)
    return rd(o * torch.sigmoid(rd(h @ P[p + "g"].T))) @ P[p + "o"].T


def dense_ff(h, P, p, rd=ident):
    return rd(gelu_tanh(rd(h @ P[p + "up"].T))) @ P[p + "down"].T


def kind_of(layer):
    head, _, tail = layer["type"].rpartition("_")
    return head if head and tail.isdigit() else layer["type"]


def forward(tokens, P, cfg, rd=ident, streams=None):
    """Logits [T, vocab] of one sequence (in a tuple, as the other plain statements return them); streams: a list that
    receives the residual stream after every layer."""
    eps, v_first = cfg["norm"]["eps"], None
    x = P["embed"][torch.tensor(tokens)] * (cfg.get("embedding") or {}).get("scale", 1.0)
    for l, L in enumerate(cfg["layers"]):
        p, m, kind = f"l{l}.", L["mixer"], kind_of(L)
        h = rd(x)
        if kind == "attention":
            mixes = m.get("v_mix", False)
            y, own = attention(h, P, p + "mix.", m, eps, v_first if mixes else None, rd)
            if mixes and v_first is None:
                v_first = own
        else:
            y = (mlstm if kind == "mlstm" else latent_attention)(h, P, p + "mix.", m, eps, rd)
        x = x + one_plus(y, P[p + "norm1"], eps)
        if L.get("mlp"):
            x = x + one_plus(dense_ff(rd(x), P, p + "mlp.", rd), P[p + "norm2"], eps)
        if streams is not None:
            streams.append(x)
    return (rd(one_plus(x, P["final.norm"], eps)) @ P["embed"].T,)
