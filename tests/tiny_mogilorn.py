"""Small Mogilorn configurations for the tests, and weights for them that make a fault visible.

The configurations differ from each other in every size, in the order and kinds of layers and in the constants; sizes
that could hide a fault by being equal (query and key/value heads, key and value sizes, turned and head sizes, inner and
model width) or by being 1 (heads, windows of one position) take both forms.  Biases, sinks and shares of mixed values are
large, norm weights far from zero.  Everything is stored in bfloat16, as a checkpoint is.
"""
import hashlib
import json
import os

import torch


def rot(dims, base, scaling=None):
    out = dict(dims=dims, base=base)
    if scaling:
        out["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return out


def attention(heads, kv_heads, dim, vdim, scale, ff, turn=None, softcap=None, v_mix=False):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, v_mix=v_mix)
    if turn:
        m["rot"] = turn
    if softcap:
        m["softcap"] = softcap
    return layer("attention", m, ff)


def mlstm(heads, dim, vdim, cap, ff):
    return layer("mlstm", dict(heads=heads, dim=dim, vdim=vdim, gate_cap=cap), ff)


def latent(heads, dim, rot_dim, vdim, kv_rank, window, scale, base, ff, scaling=None):
    m = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, scale=scale)
    if rot_dim:
        m["rot"] = rot(rot_dim, base, scaling)
    if window:
        m["mask"] = dict(size=window)
    return layer("latent_attention", m, ff)


def layer(kind, mixer, ff):
    return dict(type=kind, mixer=mixer, mlp=dict(kind="dense", ff=ff) if ff else None)


def model(vocab, width, eps, emb_scale, layers):
    return dict(architecture="Mogilorn", vocab=vocab, width=width, norm=dict(eps=eps), embedding=dict(scale=emb_scale),
                layers=layers)


# A: all mixers, the second of three attentions mixes nothing, windows shorter than a page, the order begins with a memory
TINY_A = model(150, 64, 1e-5, 3.0, [
    mlstm(3, 16, 24, 4.0, 40),
    attention(4, 2, 16, 24, 0.3, 72, rot(16, 100.0, (3.0, 1.0, 4.0, 40.0)), 6.0, True),
    latent(3, 16, 8, 24, 40, 20, 0.25, 50.0, 56),
    attention(6, 3, 24, 16, 0.25, 64, rot(8, 1000.0), 9.0, False),
    attention(2, 2, 32, 24, 0.2, 48, rot(20, 300.0, (8.0, 0.5, 3.0, 90.0)), 4.0, True),
    latent(2, 24, 4, 8, 24, 70, 0.3, 900.0, 40, (2.0, 1.0, 2.0, 30.0))])

# B: sizes that are multiples of nothing convenient; no caps, layers without feed-forward, a window of one position
TINY_B = model(77, 36, 1e-6, 1.0, [
    attention(2, 1, 12, 20, 0.4, None, rot(6, 40.0), None, True),
    latent(3, 7, 6, 9, 21, 1, 0.4, 70.0, 44),
    mlstm(1, 7, 9, 12.0, None),
    attention(3, 1, 20, 20, 0.3, 28, None, 5.0, True),
    latent(5, 12, 2, 5, 10, 65, 0.3, 10.0, None)])

# C: one head of everything, key and value sizes equal, a window of a whole page, no window, the same value channels in
# another number of heads
TINY_C = model(96, 32, 1e-6, 0.5, [
    attention(1, 1, 16, 16, 0.35, 32, rot(16, 10.0), 2.0, True),
    latent(1, 8, 8, 8, 8, 64, 0.35, 10.0, 16),
    mlstm(1, 8, 8, 2.0, 48),
    attention(4, 2, 8, 8, 0.4, 32, rot(2, 10.0), 30.0, True),
    latent(1, 8, 0, 8, 16, 0, 0.3, 10.0, 32)])

# M: sizes that the tensor-core kernels take (heads of 64 and 128, widths that are multiples of 8)
TINY_M = model(210, 128, 1e-6, 2.0, [
    attention(4, 2, 64, 64, 0.125, 256, rot(64, 1000.0, (4.0, 1.0, 4.0, 64.0)), 20.0, True),
    latent(4, 48, 16, 64, 64, 96, 0.125, 500.0, 192),
    mlstm(2, 64, 64, 15.0, 128),
    attention(2, 1, 128, 128, 0.09, 136, rot(96, 1000.0), 50.0, True),
    latent(2, 96, 32, 80, 128, 130, 0.09, 500.0, 128),
    attention(4, 2, 64, 48, 0.125, 64, rot(32, 200.0), 8.0, False)])

# L: prompts of a thousand tokens through the long-prompt attention kernels, windows that are no multiple of a tile
TINY_L = model(120, 64, 1e-6, 1.5, [
    attention(2, 1, 64, 64, 0.125, None, rot(64, 20000.0, (5.0, 1.0, 3.0, 256.0)), 15.0, True),
    latent(2, 48, 16, 64, 64, 333, 0.125, 10000.0, None),
    latent(1, 96, 32, 72, 40, 800, 0.09, 10000.0, 64),
    attention(1, 1, 128, 64, 0.09, None, rot(128, 10000.0), 40.0, True)])

# W: heads beyond the tensor-core kernels, latents of many channels, more heads than a block of the latent kernels takes
TINY_W = model(130, 96, 1e-5, 1.0, [
    attention(2, 1, 160, 144, 0.08, 80, rot(120, 5000.0), 12.0, True),
    latent(2, 112, 32, 136, 200, 90, 0.08, 700.0, 64),
    latent(19, 8, 16, 24, 264, 37, 0.2, 700.0, None),
    attention(8, 1, 20, 144, 0.2, 64, rot(20, 5000.0, (2.0, 1.0, 2.0, 128.0)), 7.0, True)])

# one mechanism at a time
ONLY_ATTENTION = model(64, 32, 1e-6, 1.0, [attention(4, 2, 16, 24, 0.3, None, rot(12, 100.0, (4.0, 1.0, 4.0, 60.0)), 3.0)])
ONLY_MIX = model(64, 32, 1e-6, 1.0, [attention(2, 1, 16, 16, 0.3, None, None, None, True), attention(2, 1, 16, 16, 0.3, None, None, None, True)])
ONLY_MLSTM = model(64, 32, 1e-6, 1.0, [mlstm(4, 16, 24, 5.0, None)])
ONLY_LATENT = model(64, 32, 1e-6, 1.0, [latent(4, 12, 8, 16, 24, 24, 0.3, 100.0, None)])
ONLY_FF = model(64, 24, 1e-6, 1.0, [latent(1, 8, 0, 8, 8, 1, 0.3, 10.0, 88)])            # a window of the present token alone

ALL = {"A": TINY_A, "B": TINY_B, "C": TINY_C, "M": TINY_M, "L": TINY_L, "W": TINY_W, "attention": ONLY_ATTENTION, "mix": ONLY_MIX,
       "mlstm": ONLY_MLSTM, "latent": ONLY_LATENT, "ff": ONLY_FF}


def _gen(seed, name):
    g = torch.Generator()
    g.manual_seed(int.from_bytes(hashlib.sha256(f"{seed}:{name}".encode()).digest()[:8], "little") & ((1 << 63) - 1))
    return g


def make_tensors(config, seed):
    """{name: bfloat16 tensor} for a configuration dict."""
    from catena_models_b200.config.registry import config_from_dict

    arch, typed = config_from_dict(config)
    scale = config["embedding"]["scale"]
    out = {}
    for spec in arch.define(typed).tensor_specs():
        g, name, shape = _gen(seed, spec.name), spec.name, tuple(spec.shape)
        n = lambda std=1.0: torch.randn(shape, generator=g) * std
        tail = name.split(".")[-1]
        if tail in ("norm1", "norm2") or name == "final.norm":
            t = n(0.3)                                              # stored as the distance from one
        elif tail == "norm":
            t = 1.0 + n(0.3)
        elif tail == "vmix":
            t = 0.35 + n(0.15)
        elif tail == "sink":
            t = n(1.5)
        elif name.endswith(".f.b"):
            t = 2.0 + n(1.5)                                        # forgets from within a few tokens to hardly at all
        elif tail == "b":
            t = n(0.7)
        elif tail in ("i", "f"):
            t = n(2.0 / shape[-1] ** 0.5)
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
