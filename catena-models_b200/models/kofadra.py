"""The Kofadra decoder as parts.

The embedding rows are multiplied by `embedding.scale`.  The residual is `streams` hyper-connected copies (float32); a layer
is a `HyperBlock`: a layer norm of the streams' weighted sum and a mixer, then (if the layer has one) the same with a
feed-forward, each written back to all streams.  Without `streams` it is a `PreNormBlock` on a plain float32 stream.  The
mixer is a gated delta rule behind short causal filters (`delta_rule`), or a grouped-query attention with normed heads, no
rotation, chunked mask and one more term of score 0 in the softmax's denominator (`gqa_attention` with `chunk` and
`sink_value`).  The feed-forward is routed (`softmax_chosen`: the weights are a softmax over the chosen experts' logits).
A loop runs layers start .. stop-1 `times` times with the same weights: the plan names the same blocks again with state
units of their own.

Tensor names: `embed`, `l<i>.norm1`, `l<i>.norm2`, `l<i>.hc{1,2}.{in,out,mix}`, `l<i>.mix.{q,k,v}{,.conv}`,
`l<i>.mix.{b,a,A_log,dt_bias,g,norm,o}` or `l<i>.mix.{q,k,v,q.norm,k.norm,o}`,
`l<i>.mlp.{router,router.b,e<j>.{gate,up,down}}`, `final.norm`, `head`.
"""
from __future__ import annotations

from ..config.kofadra import KofadraConfig
from ..config.registry import register_architecture
from ..engine.definition import ModelDefinition, PlanEntry
from ..parts import build_part
from ..parts.linear import Linear
from ..weights.loader import TensorSpec


def _mixer(cfg, i, layer):
    W, m, p = cfg.width, layer.mixer, f"l{i}.mix."
    if layer.type == "delta":
        return build_part("mixer", "delta_rule", prefix=p, hidden=W, heads=m.heads, kv_heads=m.kv_heads, dim=m.dim,
                          value_dim=m.vdim, taps=m.taps, eps=cfg.norm_eps, out_dtype="float32")
    return build_part("mixer", "gqa_attention", prefix=p, hidden=W, heads=m.heads, kv_heads=m.kv_heads, head_dim=m.dim,
                      value_dim=m.vdim, window=0, chunk=m.chunk, position=build_part("position", "none"),
                      qk_norm_eps=cfg.norm_eps, output_gate=False, scale=m.scale, sink_value=0.0,
                      names={"q": "q", "k": "k", "v": "v", "out": "o", "q_norm": "q.norm", "k_norm": "k.norm"}, out_dtype="float32")


def _feed_forward(cfg, i, mlp):
    if mlp is None:
        return None
    return build_part("feed_forward", "routed_swiglu", prefix=f"l{i}.mlp.", hidden=cfg.width, intermediate=mlp.ff,
                      experts=mlp.experts, top=mlp.top, gate="softmax_chosen", weight_on="output", bias_name="router.b")


def _norm(cfg, name, read_name=None):
    if not cfg.streams:
        return build_part("norm", "layer", name=name, width=cfg.width, eps=cfg.norm_eps)
    return build_part("norm", "streams", name=name, width=cfg.width, eps=cfg.norm_eps, streams=cfg.streams, read_name=read_name)


def _block(cfg, i, layer):
    ff, p = _feed_forward(cfg, i, layer.mlp), f"l{i}."
    parts = dict(mixer=_mixer(cfg, i, layer), feed_forward=ff, input_norm=_norm(cfg, p + "norm1", p + "hc1.in"),
                 ffn_norm=_norm(cfg, p + "norm2", p + "hc2.in") if ff is not None else None)
    if not cfg.streams:
        return build_part("block", "prenorm", **parts)
    return build_part("block", "hyper", streams=cfg.streams, mixer_tensors=(p + "hc1.mix", p + "hc1.out"),
                      ffn_tensors=(p + "hc2.mix", p + "hc2.out") if ff is not None else None, **parts)


def define(cfg: KofadraConfig) -> ModelDefinition:
    return ModelDefinition(
        architecture=cfg.architecture, vocab_size=cfg.vocab, hidden_size=cfg.width, embedding_name="embed",
        blocks=[_block(cfg, i, layer) for i, layer in enumerate(cfg.layers)],
        plan=[PlanEntry(block=layer, state=unit) for unit, layer in enumerate(cfg.run_order())],      # every run has its own state
        final_norm=_norm(cfg, "final.norm"), head=Linear("head", cfg.vocab, cfg.width),
        extra_tensors=tuple(TensorSpec(name, shape, "vector") for name, shape in cfg.unused),
        embedding_scale=cfg.embedding_scale, residual_float32=True, streams=cfg.streams)


register_architecture("Kofadra", KofadraConfig, define)
