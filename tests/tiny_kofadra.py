"""Small Kofadra configurations for the tests, and weights for them that make a fault visible.

The configurations differ from each other in every size, in the order and kinds of layers and in the constants; sizes
that could hide a fault by being equal (query and key/value heads, key and value sizes, expert and model width) or by
being 1 (heads, streams, top, taps, chunks of one position, passes of the loop) take both forms.  Decays reach from
"keeps almost everything" to "forgets within a few tokens"; stream mixes are far from the identity; router biases are
large enough to change the choice of experts.  Everything is stored in bfloat16, as a checkpoint is.
"""
import hashlib
import json
import os

import torch


def delta(heads, kv_heads, dim, vdim, conv, mlp):
    return dict(type="delta", mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv), mlp=mlp)


def attention(heads, kv_heads, dim, vdim, chunk, scale, mlp):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale)
    if chunk:
        m["mask"] = dict(size=chunk)
    return dict(type="attention", mixer=m, mlp=mlp)


def moe(ff, experts, top):
    return dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top))


def model(vocab, width, eps, emb_scale, streams, layers, loop=None):
    return dict(architecture="Kofadra", vocab=vocab, width=width, norm=dict(eps=eps), embedding=dict(scale=emb_scale),
                streams=streams, layers=layers, **(dict(loop=dict(start=loop[0], stop=loop[1], times=loop[2])) if loop else {}))


# A: both mixers twice, fewer key/value heads than heads, chunks shorter than a page, the middle layers run three times
TINY_A = model(150, 64, 1e-5, 3.0, 3, [
    delta(4, 2, 16, 24, 4, moe(40, 6, 2)),
    attention(4, 2, 16, 16, 20, 0.3, moe(24, 4, 3)),
    delta(2, 2, 24, 8, 2, moe(32, 5, 1)),
    attention(3, 3, 16, 16, 50, 0.25, moe(24, 4, 2))], loop=(1, 3, 3))

# B: sizes that are multiples of nothing convenient; padded heads with a head norm; one stream; layers without feed-forward;
# one tap; no loop
TINY_B = model(77, 36, 1e-6, 1.0, 1, [
    attention(2, 1, 12, 20, 7, 0.4, None),
    delta(3, 1, 7, 9, 1, moe(20, 3, 3)),
    attention(3, 3, 20, 12, 70, 0.3, moe(28, 7, 4)),
    delta(1, 1, 5, 12, 5, None)])

# C: one head of everything, one expert, chunks of whole pages, no chunks, key and value sizes equal; a loop over everything
TINY_C = model(96, 32, 1e-6, 0.5, 2, [
    delta(1, 1, 8, 8, 3, moe(16, 1, 1)),
    attention(1, 1, 8, 8, 64, 0.35, None),
    attention(4, 1, 8, 16, 0, 0.3, moe(16, 4, 4))], loop=(0, 3, 2))

# M: sizes that the tensor-core kernels take (heads of 64 and 128, widths that are multiples of 8)
TINY_M = model(210, 128, 1e-6, 2.0, 4, [
    delta(4, 2, 64, 128, 4, moe(64, 8, 2)),
    attention(4, 2, 64, 64, 96, 0.125, moe(64, 6, 3)),
    attention(2, 1, 128, 128, 130, 0.09, moe(72, 4, 1)),
    delta(2, 1, 128, 64, 3, moe(64, 8, 4))], loop=(2, 4, 1))

# L: chunks of hundreds of tokens (the long-prompt attention kernels), one that is no multiple of a tile
TINY_L = model(120, 64, 1e-6, 1.5, 2, [
    attention(2, 1, 64, 64, 800, 0.125, None),
    attention(2, 2, 64, 64, 333, 0.125, None)])

# one mechanism at a time
ONLY_DELTA = model(64, 32, 1e-6, 1.0, 1, [delta(4, 2, 16, 24, 4, None)])
ONLY_ATTENTION = model(64, 32, 1e-6, 1.0, 1, [attention(4, 2, 16, 24, 24, 0.3, None)])
ONLY_MOE = model(64, 24, 1e-6, 1.0, 1, [attention(1, 1, 8, 8, 1, 0.3, moe(40, 8, 3))])       # chunks of one position
ONLY_STREAMS = model(64, 24, 1e-6, 2.0, 5, [attention(1, 1, 8, 8, 2, 0.3, moe(8, 2, 1))], loop=(0, 1, 4))

ALL = {"A": TINY_A, "B": TINY_B, "C": TINY_C, "M": TINY_M, "L": TINY_L, "delta": ONLY_DELTA, "attention": ONLY_ATTENTION,
       "moe": ONLY_MOE, "streams": ONLY_STREAMS}


def _gen(seed, name):
    g = torch.Generator()
    g.manual_seed(int.from_bytes(hashlib.sha256(f"{seed}:{name}".encode()).digest()[:8], "little") & ((1 << 63) - 1))
    return g


def make_tensors(config, seed):
    """{name: bfloat16 tensor} for a configuration dict."""
    from catena_models_b200.config.registry import config_from_dict

    arch, typed = config_from_dict(config)
    scale, S = config["embedding"]["scale"], config["streams"]
    out = {}
    for spec in arch.define(typed).tensor_specs():
        g, name, shape = _gen(seed, spec.name), spec.name, tuple(spec.shape)
        n = lambda std=1.0: torch.randn(shape, generator=g) * std
        tail = name.split(".")[-1]
        if tail in ("norm1", "norm2", "norm"):
            t = 1.0 + n(0.2)
        elif tail == "conv":
            t = n(0.6)
        elif tail == "A_log":
            t = torch.rand(shape, generator=g) * 4.0 - 3.0          # rates from 0.05 to 2.7
        elif tail == "dt_bias":
            t = n(1.0)
        elif name.endswith("router.b"):
            t = n(0.8)
        elif tail == "router":
            t = n(2.0 / shape[-1] ** 0.5)
        elif ".hc" in name and tail == "in":
            t = 1.0 / S + n(0.3)
        elif ".hc" in name and tail == "out":
            t = 1.0 + n(0.3)
        elif ".hc" in name and tail == "mix":
            t = 0.6 * torch.eye(S) + 0.4 / S + n(0.15)
        elif name == "embed":
            t = n(1.0 / scale)
        else:
            t = n(1.0 / shape[-1] ** 0.5)
        out[name] = t.to(torch.bfloat16)
    return out


def make_folder(tmp, name, seed=0, config=None, tensors=None):
    from catena_models_b200.weights.safetensors_io import write_safetensors

    config = config or ALL[name]
    folder = os.path.join(str(tmp), name)
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as fh:
        json.dump(config, fh)
    write_safetensors(os.path.join(folder, "model.safetensors"), tensors or make_tensors(config, seed))
    return folder


def load_plain(folder):
    """(config dict, {name: float64 tensor}) as the plain implementation takes them."""
    from catena_models_b200.weights.safetensors_io import SafetensorsFile

    with open(os.path.join(folder, "config.json")) as fh:
        cfg = json.load(fh)
    f = SafetensorsFile(os.path.join(folder, "model.safetensors"))
    tensors = {n: f.tensor(n).clone().to(torch.float64) for n in f.names()}
    f.close()
    return cfg, tensors


def prompt(n, vocab, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, vocab, (n,), generator=g).tolist()
