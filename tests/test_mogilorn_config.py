"""Reading a Mogilorn config.json: every size and constant lands in the typed configuration, what may be left out gets its
neutral value, what contradicts itself or the kernels' limits is refused when the file is read, and the definition names exactly
the tensors that the layers need.  The rotation's rates against the plain statement."""
import copy

import pytest
import torch

import plain_mogilorn as plain
import tiny_mogilorn as tiny
from catena_models_b200.config.base import ConfigError
from catena_models_b200.config.registry import config_from_dict


def specs_of(config):
    arch, cfg = config_from_dict(config)
    return {s.name: tuple(s.shape) for s in arch.define(cfg).tensor_specs()}


def test_fields_of_every_layer():
    arch, cfg = config_from_dict(tiny.TINY_A)
    assert arch.name == "Mogilorn"
    assert (cfg.vocab, cfg.width, cfg.norm_eps, cfg.embedding_scale) == (150, 64, 1e-5, 3.0)
    s, a, l = cfg.layers[:3]
    assert (s.type, s.mixer.heads, s.mixer.dim, s.mixer.vdim, s.mixer.gate_cap, s.mlp.ff) == ("mlstm", 3, 16, 24, 4.0, 40)
    m = a.mixer
    assert (a.type, m.heads, m.kv_heads, m.dim, m.vdim, m.scale, m.softcap, m.v_mix) == ("attention", 4, 2, 16, 24, 0.3, 6.0, True)
    assert (m.rot.dims, m.rot.base) == (16, 100.0)
    assert (m.rot.scaling.factor, m.rot.scaling.low, m.rot.scaling.high, m.rot.scaling.original) == (3.0, 1.0, 4.0, 40.0)
    m = l.mixer
    assert (m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank, m.window, m.scale) == (3, 16, 8, 24, 40, 20, 0.25)
    assert (m.rot.dims, m.rot.base, m.rot.scaling) == (8, 50.0, None)
    assert cfg.value_source() == 1 and not cfg.layers[3].mixer.v_mix


def test_what_may_be_left_out():
    short = copy.deepcopy(tiny.ONLY_ATTENTION)
    del short["embedding"]
    for key in ("kv_heads", "vdim", "softcap", "rot", "v_mix"):
        del short["layers"][0]["mixer"][key]
    _, c = config_from_dict(short)
    m = c.layers[0].mixer
    assert (c.embedding_scale, m.kv_heads, m.vdim, m.softcap, m.rot, m.v_mix) == (1.0, 4, 16, 0.0, None, False)
    assert c.value_source() is None and c.layers[0].mlp is None
    _, c = config_from_dict(tiny.TINY_C)
    assert c.layers[4].mixer.window == 0 and c.layers[4].mixer.rot is None
    numbered = copy.deepcopy(tiny.ONLY_MLSTM)
    numbered["layers"][0]["type"] = "mlstm_2"
    assert config_from_dict(numbered)[1].layers[0].type == "mlstm"


def test_the_definition_names_the_layers_tensors():
    a = specs_of(tiny.TINY_A)
    assert a["l1.mix.q"] == (64, 64) and a["l1.mix.k.b"] == (32,) and a["l1.mix.v.b"] == (48,) and a["l1.mix.o.b"] == (64,)
    assert a["l1.mix.g"] == (96, 64) and a["l1.mix.o"] == (64, 96) and a["l1.mix.q.norm"] == (16,) and a["l1.mix.vmix"] == ()
    assert "l3.mix.vmix" not in a and a["l4.mix.vmix"] == ()
    assert a["l2.mix.q"] == (72, 64) and a["l2.mix.dkv"] == (48, 64) and a["l2.mix.dkv.norm"] == (40,)
    assert a["l2.mix.uk"] == (48, 40) and a["l2.mix.uv"] == (72, 40) and a["l2.mix.sink"] == (3,) and a["l2.mix.g"] == (72, 64)
    assert a["l0.mix.i.b"] == (3,) and a["l0.mix.norm"] == (72,)
    assert a["l5.mlp.up"] == (40, 64) and a["l5.mlp.down"] == (64, 40) and a["embed"] == (150, 64) and "head" not in a
    b = specs_of(tiny.TINY_B)
    assert not any(n.startswith(("l0.mlp", "l0.norm2")) for n in b)
    assert b["l0.mix.q.norm"] == (12,) and b["l0.mix.v"] == (20, 36) and b["l0.mix.o"] == (36, 40)       # stored sizes, not padded ones


def test_tensors_that_nothing_reads_are_no_surprise():
    arch, cfg = config_from_dict(tiny.TINY_B)
    more = cfg.with_tensor_shapes({"l0.norm2": (36,), "l1.norm2": (36,)})
    assert more.unused == (("l0.norm2", (36,)),)
    assert any(s.name == "l0.norm2" for s in arch.define(more).tensor_specs())
    more = config_from_dict(tiny.ONLY_ATTENTION)[1].with_tensor_shapes({"l0.mix.vmix": ()})
    assert more.unused == (("l0.mix.vmix", ()),)


@pytest.mark.parametrize("change", [
    lambda l: l[1]["mixer"].update(kv_heads=3),                            # heads that do not divide
    lambda l: l[1]["mixer"].update(dim=300),                               # beyond the attention kernels
    lambda l: l[1]["mixer"]["rot"].update(dims=18),                        # more turned channels than the head has
    lambda l: l[1]["mixer"]["rot"].update(dims=7),
    lambda l: l[1]["mixer"]["rot"]["scaling"].update(high=0.5),
    lambda l: l[1]["mixer"].update(softcap=-1.0),
    lambda l: l[4]["mixer"].update(vdim=20),                               # mixes values of another size
    lambda l: l[2]["mixer"].update(kv_rank=600),
    lambda l: l[2]["mixer"]["rot"].update(dims=10),
    lambda l: l[0]["mixer"].update(dim=2000),
    lambda l: l[0]["mixer"].pop("gate_cap"),
    lambda l: l[0].update(type="mamba"),
    lambda l: l[0]["mlp"].update(kind="moe"),
    lambda l: l[2]["mixer"].pop("kv_rank")])
def test_refused_when_the_file_is_read(change):
    config = copy.deepcopy(tiny.TINY_A)
    change(config["layers"])
    with pytest.raises(ConfigError):
        config_from_dict(config)


@pytest.mark.parametrize("scaling", [(6.0, 1.0, 5.0, 700.0), (8.0, 1.0, 4.0, 8192.0), (2.0, 0.5, 3.0, 33.0)])
@pytest.mark.parametrize("dims, base", [(64, 10000.0), (128, 500000.0), (12, 30.0)])
def test_rates_rescaled_by_wavelength(dims, base, scaling):
    from catena_models_b200.parts import build_part

    spec = tiny.rot(dims, base, scaling)
    part = build_part("position", "wavelength_rotary", dims=dims, theta=base, **spec["scaling"])
    want = plain.rotation_rates(spec)
    assert torch.allclose(torch.tensor(part.rates, dtype=torch.float64), want, rtol=1e-12, atol=0.0)
    plain_rates = plain.rotation_rates(tiny.rot(dims, base))
    assert float((want / plain_rates).max()) == 1.0                        # the fastest pair keeps its rate
    assert part.pairing == "interleaved" and part.magnitude == 1.0
