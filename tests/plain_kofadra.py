"""Plain statement of the Kofadra decoder, one function per mechanism, in float64 on the CPU.

Nothing here is shared with the library: the tests compare the engine's kernels with these functions.  `P` is
{tensor name: float64 tensor}; `cfg` is the dict of config.json; h [T, W] are the rows of one sequence from position 0.

    layer_norm(x)     (x - mean(x)) / sqrt(mean((x - mean(x))^2) + eps) * w
    streams           X_s = E[token] * s_e for every stream s
    sublayer          y = f(layer_norm(sum_s a_s X_s));  X_t <- sum_s M_st X_s + c_t y   (a, M, c of the sublayer)
    output            layer_norm(sum_s X_s) H^T

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


def silu(z):
    return z * torch.sigmoid(z)


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x, w, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w


def stream_read(X, a):
    """X [S, T, W], a [S] -> sum_s a_s X_s."""
    return (a[:, None, None] * X).sum(0)


def stream_write(X, M, c, y):
    """X_t <- sum_s M[s, t] X_s + c_t y, all t from the old X."""
    return torch.stack([sum(M[s, t] * X[s] for s in range(X.shape[0])) + c[t] * y for t in range(X.shape[0])])


def taps(u, w):
    """y_t = sum_j w[:, j] u_(t - K + 1 + j) per channel, zeros before the first row.  u [T, C], w [C, K]."""
    T, K = u.shape[0], w.shape[1]
    full = torch.cat([torch.zeros(K - 1, u.shape[1], dtype=u.dtype), u])
    return sum(w[:, j] * full[j:j + T] for j in range(K))


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_rule(q, k, v, beta, g, S=None):
    """q, k [T, H, D], v [T, H, DV], beta, g [T, H]; S [H, D, DV] or None (zeros).  Per token and head: S <- g S;
    u = beta (v - S^T k); S <- S + k u^T; o = S^T q.  Returns (o [T, H, DV], S)."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[2], dtype=F64) if S is None else S.clone()
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for t in range(T):
        S = g[t, :, None, None] * S
        u = beta[t, :, None] * (v[t] - (S * k[t, :, :, None]).sum(1))
        S = S + k[t, :, :, None] * u[:, None, :]
        out[t] = (S * q[t, :, :, None]).sum(1)
    return out, S


def delta_inputs(h, P, p, m, rd=ident):
    """(q, k, v, beta, g) of every head, as delta_rule takes them."""
    T = h.shape[0]
    H, G, D, DV = m["heads"], m.get("kv_heads", m["heads"]), m["dim"], m.get("vdim", m["dim"])
    rows = {s: rd(silu(taps(rd(h @ P[p + s].T), P[f"{p}{s}.conv"]))) for s in "qkv"}
    spread = lambda x: x.repeat_interleave(H // G, 1)
    q = spread(unit(rows["q"].view(T, G, D))) / math.sqrt(D)
    k = spread(unit(rows["k"].view(T, G, D)))
    beta = torch.sigmoid(h @ P[p + "b"].T)
    z = h @ P[p + "a"].T + P[p + "dt_bias"]
    g = torch.exp(-torch.exp(P[p + "A_log"]) * (torch.clamp(z, min=0) + torch.log1p(torch.exp(-torch.abs(z)))))
    return q, k, rows["v"].view(T, H, DV), beta, g


def delta_mixer(h, P, p, m, eps, rd=ident):
    T = h.shape[0]
    q, k, v, beta, g = delta_inputs(h, P, p, m, rd)
    o, _ = delta_rule(q, k, v, beta, g)
    o = rms(o, eps) * P[p + "norm"] * silu(rd(h @ P[p + "g"].T)).view(T, m["heads"], -1)
    return rd(o.reshape(T, -1)) @ P[p + "o"].T


def sees(i, j, size):
    """True if position i may look at position j: j is not later, and in the same chunk of `size` (0: no chunks)."""
    return j <= i and (not size or i // size == j // size)


def sink_softmax(s):
    """exp(s_j) / (1 + sum_j exp(s_j)): one more term of score 0, without a value."""
    mx = max(float(s.max()), 0.0)
    e = torch.exp(s - mx)
    return e / (math.exp(-mx) + e.sum())


def chunk_attention(h, P, p, m, eps, rd=ident):
    T = h.shape[0]
    H, G, D, DV = m["heads"], m.get("kv_heads", m["heads"]), m["dim"], m.get("vdim", m["dim"])
    size = (m.get("mask") or {}).get("size", 0)
    q = rd(rms(rd(h @ P[p + "q"].T).view(T, H, D), eps) * P[p + "q.norm"])
    k = rd(rms(rd(h @ P[p + "k"].T).view(T, G, D), eps) * P[p + "k.norm"])
    v = rd(h @ P[p + "v"].T).view(T, G, DV)
    out = torch.zeros(T, H, DV, dtype=F64)
    for i in range(T):
        seen = [j for j in range(T) if sees(i, j, size)]
        for hh in range(H):
            g = hh // (H // G)
            out[i, hh] = sink_softmax((k[seen, g] @ q[i, hh]) * m["scale"]) @ v[seen, g]
    return rd(out.reshape(T, H * DV)) @ P[p + "o"].T


def expert(h, P, p, rd=ident):
    return rd(silu(rd(h @ P[p + "gate"].T)) * rd(h @ P[p + "up"].T)) @ P[p + "down"].T


def route(h, P, p, r, ids=None):
    """(chosen experts [T, top], their weights [T, top]); `ids`: the choice to use instead of the router's own."""
    z = h @ P[p + "router"].T + P[p + "router.b"]
    if ids is None:
        order = [sorted(range(z.shape[1]), key=lambda e: (-float(z[t, e]), e))[:r["top"]] for t in range(z.shape[0])]
        ids = torch.tensor(order, dtype=torch.long)
    return ids, torch.softmax(z.gather(1, ids), -1)


def moe_ff(h, P, p, f, rd=ident, ids=None):
    ids, wts = route(h, P, p, f["router"], ids)
    out = torch.zeros_like(h)
    for e in sorted(set(ids.flatten().tolist())):
        t, j = torch.nonzero(ids == e, as_tuple=True)
        out[t] += wts[t, j, None] * expert(h[t], P, f"{p}e{e}.", rd)
    return out, ids


def run_order(cfg):
    """Layer indices in the order they run."""
    L, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(L))
    body = list(range(loop["start"], loop["stop"]))
    return list(range(loop["start"])) + body * loop["times"] + list(range(loop["stop"], L))


def forward(tokens, P, cfg, rd=ident, expert_ids=None, ids_out=None, streams=None):
    """Logits [T, vocab] of one sequence (in a tuple, as the other plain statements return them).  expert_ids: {run:
    ids} to pin every router's choice (runs count layer executions); ids_out: a dict that receives the choices made;
    streams: a list that receives the sum of the streams after every layer run."""
    eps = cfg["norm"]["eps"]
    e = P["embed"][torch.tensor(tokens)] * (cfg.get("embedding") or {}).get("scale", 1.0)
    X = torch.stack([e] * cfg["streams"])
    for run, i in enumerate(run_order(cfg)):
        p, L = f"l{i}.", cfg["layers"][i]

        def sublayer(X, q, f):
            y = f(rd(layer_norm(stream_read(X, P[f"{p}hc{q}.in"]), P[f"{p}norm{q}"], eps)))
            return stream_write(X, P[f"{p}hc{q}.mix"], P[f"{p}hc{q}.out"], y)

        mixer = delta_mixer if L["type"].startswith("delta") else chunk_attention
        X = sublayer(X, 1, lambda n: mixer(n, P, p + "mix.", L["mixer"], eps, rd))
        if L.get("mlp"):
            def ff(n):
                y, ids = moe_ff(n, P, p + "mlp.", L["mlp"], rd, (expert_ids or {}).get(run))
                if ids_out is not None:
                    ids_out[run] = ids
                return y
            X = sublayer(X, 2, ff)
        if streams is not None:
            streams.append(X.sum(0))
    return (rd(layer_norm(X.sum(0), P["final.norm"], eps)) @ P["head"].T,)
