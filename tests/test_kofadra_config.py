"""Reading a Kofadra config.json: every size and constant lands in the typed configuration, what may be left out gets
its neutral value, what the kernels cannot run or what contradicts itself is refused when the file is read, and the
definition names exactly the tensors that the layers need, in the order in which the loop runs them."""
import copy

import pytest

import tiny_kofadra as tiny
from catena_models_b200.config.base import ConfigError
from catena_models_b200.config.registry import config_from_dict


def specs_of(config):
    arch, cfg = config_from_dict(config)
    return {s.name: tuple(s.shape) for s in arch.define(cfg).tensor_specs()}


def test_fields_of_every_layer():
    arch, cfg = config_from_dict(tiny.TINY_A)
    assert arch.name == "Kofadra"
    assert (cfg.vocab, cfg.width, cfg.norm_eps, cfg.embedding_scale, cfg.streams) == (150, 64, 1e-5, 3.0, 3)
    d, a, d2, a2 = cfg.layers
    m = d.mixer
    assert (d.type, m.heads, m.kv_heads, m.dim, m.vdim, m.taps) == ("delta", 4, 2, 16, 24, 4)
    assert (d.mlp.ff, d.mlp.experts, d.mlp.top) == (40, 6, 2)
    m = a.mixer
    assert (a.type, m.heads, m.kv_heads, m.dim, m.vdim, m.chunk, m.scale) == ("attention", 4, 2, 16, 16, 20, 0.3)
    assert (cfg.loop.start, cfg.loop.stop, cfg.loop.times) == (1, 3, 3)
    assert cfg.run_order() == [0, 1, 2, 1, 2, 1, 2, 3]


def test_what_may_be_left_out():
    _, c = config_from_dict(tiny.TINY_C)
    assert c.layers[2].mixer.chunk == 0 and c.layers[1].mlp is None
    _, b = config_from_dict(tiny.TINY_B)
    assert b.loop is None and b.run_order() == [0, 1, 2, 3] and b.layers[1].mixer.taps == 1
    short = copy.deepcopy(tiny.ONLY_ATTENTION)
    del short["embedding"]
    del short["layers"][0]["mixer"]["kv_heads"], short["layers"][0]["mixer"]["vdim"]
    _, s = config_from_dict(short)
    assert s.embedding_scale == 1.0 and (s.layers[0].mixer.kv_heads, s.layers[0].mixer.vdim) == (4, 16)
    numbered = copy.deepcopy(tiny.ONLY_DELTA)
    numbered["layers"][0]["type"] = "delta_2"
    assert config_from_dict(numbered)[1].layers[0].type == "delta"


def test_the_definition_names_the_layers_tensors():
    names = specs_of(tiny.TINY_A)
    assert names["l0.mix.q.conv"] == (32, 4) and names["l0.mix.v.conv"] == (96, 4) and names["l0.mix.norm"] == (24,)
    assert names["l0.mix.b"] == names["l0.mix.a"] == (4, 64) and names["l0.mix.A_log"] == names["l0.mix.dt_bias"] == (4,)
    assert names["l1.mix.q.norm"] == (16,) and names["l1.mix.o"] == (64, 64) and "l1.mix.g" not in names
    assert names["l0.hc1.mix"] == (3, 3) and names["l0.hc2.in"] == (3,) and names["l0.hc2.out"] == (3,)
    assert names["l0.mlp.router.b"] == (6,) and names["l0.mlp.e5.down"] == (64, 40)
    assert names["final.norm"] == (64,) and names["head"] == (150, 64)
    b = specs_of(tiny.TINY_B)
    assert not any(n.startswith(("l0.mlp", "l0.hc2", "l0.norm2")) for n in b)
    assert b["l0.mix.q.norm"] == (12,) and b["l0.mix.v"] == (20, 36) and b["l0.mix.o"] == (36, 40)       # stored sizes, not padded ones


def test_every_pass_of_the_loop_has_a_state_of_its_own():
    arch, cfg = config_from_dict(tiny.TINY_A)
    plan = arch.define(cfg).plan
    assert [e.block for e in plan] == cfg.run_order() and [e.state for e in plan] == list(range(8))
    assert all(e.owns_state for e in plan)


def test_a_plain_residual_without_streams():
    plain = copy.deepcopy(tiny.TINY_A)
    del plain["streams"]
    names = specs_of(plain)
    assert not any(".hc" in n for n in names)
    arch, cfg = config_from_dict(plain)
    assert arch.define(cfg).streams == 0


def test_tensors_that_a_layer_without_feed_forward_carries_all_the_same():
    arch, cfg = config_from_dict(tiny.TINY_B)
    shapes = dict(specs_of(tiny.TINY_B), **{"l0.norm2": (36,), "l0.hc2.in": (1,)})
    names = {s.name for s in arch.define(cfg.with_tensor_shapes(shapes)).tensor_specs()}
    assert names == set(shapes)


def _with(path, value, base=None):
    cfg = copy.deepcopy(base or tiny.TINY_A)
    node = cfg
    for key in path[:-1]:
        node = node[key]
    node[path[-1]] = value
    return cfg


@pytest.mark.parametrize("path, value, text", [
    (("layers", 0, "mixer", "kv_heads"), 3, "kv_heads"),
    (("layers", 1, "mixer", "kv_heads"), 3, "kv_heads"),
    (("layers", 0, "mixer", "conv"), 99, "taps"),
    (("layers", 0, "mixer", "conv"), 0, "conv"),
    (("layers", 0, "mixer", "dim"), 2048, "key channels"),
    (("layers", 1, "mixer", "vdim"), 300, "attention heads"),
    (("layers", 1, "mixer", "scale"), 0.0, "scale"),
    (("layers", 0, "mlp", "router", "top"), 7, "top"),
    (("layers", 0, "mlp", "kind"), "dense", "known"),
    (("layers", 0, "type"), "mlstm", "known mixers"),
    (("loop", "stop"), 5, "loop"),
    (("loop", "times"), 0, "times"),
    (("streams",), 9, "streams"),
    (("norm", "eps"), 0, "eps"),
    (("width",), "wide", "integer"),
])
def test_refused_when_read(path, value, text):
    with pytest.raises(ConfigError) as e:
        config_from_dict(_with(path, value))
    assert text in str(e.value)


def test_the_mask_reaches_the_kernels_as_chunks_and_the_cache_as_a_ring():
    from catena_models_b200.cache.spec import KVStateSpec

    arch, cfg = config_from_dict(tiny.TINY_A)
    mixer = arch.define(cfg).blocks[1].mixer
    assert mixer.mask == -20 and mixer.state_spec() == KVStateSpec(2, 16, 20)
    _, c = config_from_dict(tiny.TINY_C)
    mixer = arch.define(c).blocks[2].mixer
    assert mixer.mask == 0 and mixer.state_spec() == KVStateSpec(1, 16, 0)                  # key heads padded to the values' size
