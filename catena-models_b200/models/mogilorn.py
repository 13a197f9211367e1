"""The Mogilorn decoder as parts.

The embedding rows are multiplied by `embedding.scale`; the same table, without that factor, gives the logits.  A layer is an
`OutputNormBlock` on a float32 stream: the mixer reads the stream, an RMS norm (stored as the weight's distance from one)
stands on what it adds, and the same for the feed-forward.  The mixer is a grouped-query attention with biases, normed query
and key heads, a rotation of neighbouring channels with rates rescaled by their wavelength, capped scores, values mixed with
the first such layer's, and an output gate per channel (`gqa_attention`); a matrix memory (`matrix_memory`); or an attention
over cached latents with queries straight from the input, a sliding window, a sink and a gate per channel
(`latent_attention`).  The feed-forward is a plain one with the tanh form of gelu, or none.

Tensor names: `embed`, `l<i>.norm1`, `l<i>.norm2`, `l<i>.mix.{q,k,v,o}` with `.b` for each, `l<i>.mix.{q.norm,k.norm,vmix,g}`,
or `l<i>.mix.{q,k,v,g,o,norm,i,i.b,f,f.b}`, or `l<i>.mix.{q,dkv,dkv.norm,uk,uv,sink,g,o}`, `l<i>.mlp.{up,down}`, `final.norm`.
"""
from __future__ import annotations

from ..config.mogilorn import MogilornConfig
from ..config.registry import register_architecture
from ..engine.definition import ModelDefinition, PlanEntry
from ..parts import build_part
from ..weights.loader import TensorSpec


def _position(rot):
    if rot is None:
        return build_part("position", "none")
    if rot.scaling is None:
        return build_part("position", "paired_rotary", dims=rot.dims, theta=rot.base)
    s = rot.scaling
    return build_part("position", "wavelength_rotary", dims=rot.dims, theta=rot.base, factor=s.factor, low=s.low, high=s.high,
                      original=s.original)


def _mixer(cfg, i, layer):
    W, m, p, eps = cfg.width, layer.mixer, f"l{i}.mix.", cfg.norm_eps
    if layer.type == "attention":
        mix = ("source" if i == cfg.value_source() else "mix", p + "vmix") if m.v_mix else None
        return build_part("mixer", "gqa_attention", prefix=p, hidden=W, heads=m.heads, kv_heads=m.kv_heads, head_dim=m.dim,
                          value_dim=m.vdim, window=0, position=_position(m.rot), qk_norm_eps=eps, output_gate=True,
                          gate_channels=True, scale=m.scale, softcap=m.softcap, bias=True, value_mix=mix,
                          names={"q": "q", "k": "k", "v": "v", "gate": "g", "out": "o", "q_norm": "q.norm", "k_norm": "k.norm",
                                 "q_bias": "q.b", "k_bias": "k.b", "v_bias": "v.b", "out_bias": "o.b"}, out_dtype="float32")
    if layer.type == "mlstm":
        return build_part("mixer", "matrix_memory", prefix=p, hidden=W, heads=m.heads, dim=m.dim, value_dim=m.vdim,
                          gate_cap=m.gate_cap, eps=eps, out_dtype="float32")
    return build_part("mixer", "latent_attention", prefix=p, hidden=W, heads=m.heads, dim=m.dim, rot_dim=m.rot_dim,
                      value_dim=m.vdim, kv_rank=m.kv_rank, q_rank=None, position=_position(m.rot), scale=m.scale, eps=eps,
                      output_gate=True, gate_channels=True, window=m.window, sink_name="sink", out_dtype="float32")


def _block(cfg, i, layer):
    norm = lambda name: _norm(cfg, f"l{i}.{name}")
    ff = None
    if layer.mlp is not None:
        ff = build_part("feed_forward", "gelu_tanh", prefix=f"l{i}.mlp.", hidden=cfg.width, intermediate=layer.mlp.ff,
                        out_dtype="float32")
    return build_part("block", "outnorm", mixer=_mixer(cfg, i, layer), feed_forward=ff, mixer_norm=norm("norm1"),
                      ffn_norm=norm("norm2") if ff is not None else None)


def _norm(cfg, name):
    return build_part("norm", "rms", name=name, width=cfg.width, eps=cfg.norm_eps, weight_offset=1.0)


def define(cfg: MogilornConfig) -> ModelDefinition:
    return ModelDefinition(
        architecture=cfg.architecture, vocab_size=cfg.vocab, hidden_size=cfg.width, embedding_name="embed",
        blocks=[_block(cfg, i, layer) for i, layer in enumerate(cfg.layers)],
        plan=[PlanEntry(block=i, state=i) for i in range(len(cfg.layers))], final_norm=_norm(cfg, "final.norm"), head=None,
        extra_tensors=tuple(TensorSpec(name, shape, "vector") for name, shape in cfg.unused),
        embedding_scale=cfg.embedding_scale, residual_float32=True)


register_architecture("Mogilorn", MogilornConfig, define)
