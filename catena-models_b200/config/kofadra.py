"""Configuration of the Kofadra decoder.

config.json is nested: `vocab`, `width`, `norm.eps`, `embedding.scale` (the factor on every embedding row), `streams` (how
many hyper-connected copies the residual has; absent: a plain residual); `layers`, a list whose entries give `type` (which
mixer the layer has), `mixer` (its sizes and constants) and `mlp` (the feed-forward, or null for none); `loop` (or null):
layers start .. stop-1 run `times` times in a row with the same weights, each pass with a state of its own.

Mixer types: `delta` (`heads`, `kv_heads`, `dim`, `vdim`, `conv`: taps of the short filter) and `attention` (`heads`,
`kv_heads`, `dim`, `vdim`, `scale`, `mask.size`: chunks of that many positions; absent: no chunks).  A type may carry a
numeric suffix.  Feed-forward kind: `moe` (`expert.ff`, `router.experts`, `router.top`).
"""
from __future__ import annotations

import dataclasses

from ..csrc import limits
from .base import ConfigError, Reader, base_type, section

MIXER_TYPES = ("delta", "attention")
MLP_KINDS = ("moe",)
MAX_STREAMS = 8            # csrc/hyper.cu


@dataclasses.dataclass(frozen=True)
class DeltaConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int


@dataclasses.dataclass(frozen=True)
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: int             # 0: every earlier position is seen


@dataclasses.dataclass(frozen=True)
class MlpConfig:
    ff: int
    experts: int
    top: int


@dataclasses.dataclass(frozen=True)
class LayerConfig:
    type: str
    mixer: object
    mlp: object            # MlpConfig or None


@dataclasses.dataclass(frozen=True)
class LoopConfig:
    start: int
    stop: int
    times: int


@dataclasses.dataclass(frozen=True)
class KofadraConfig:
    architecture: str
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    streams: int           # 0: a plain residual
    layers: tuple
    loop: object           # LoopConfig or None
    unused: tuple = ()     # (name, shape) of tensors that a layer without feed-forward carries all the same
    raw: dict = dataclasses.field(compare=False, default=None)

    @classmethod
    def from_dict(cls, data, where="config.json"):
        r = Reader(data, where)
        arch = r.string("architecture")
        vocab, width = r.integer("vocab", minimum=1), r.integer("width", minimum=1)
        streams = r.integer("streams", default=0, minimum=0)
        norm = section(r, data, "norm", "")
        eps = norm.number("eps", positive=True) if norm else None
        emb = section(r, data, "embedding", "", required=False)
        emb_scale = emb.number("scale", default=1.0) if emb else 1.0
        raw_layers = data.get("layers")
        if not isinstance(raw_layers, list) or not raw_layers:
            r.problem("'layers' must be a non-empty list")
            raw_layers = []
        layers = [cls._layer(r, entry, f"layers[{i}].") for i, entry in enumerate(raw_layers)]
        loop = None
        lr = section(r, data, "loop", "", required=False)
        if lr:
            loop = LoopConfig(lr.integer("start", minimum=0), lr.integer("stop", minimum=1), lr.integer("times", minimum=1))
        r.finish()
        cfg = cls(arch, vocab, width, eps, emb_scale, streams, tuple(layers), loop, raw=data)
        cfg.validate(where)
        return cfg

    @staticmethod
    def _layer(r, entry, where):
        if not isinstance(entry, dict) or not isinstance(entry.get("type"), str):
            r.problem(f"'{where}type' must be a string")
            return None
        kind = base_type(entry["type"])
        if kind not in MIXER_TYPES:
            r.problem(f"'{where}type' is '{entry['type']}'; known mixers: {', '.join(MIXER_TYPES)}")
            return None
        m = section(r, entry, "mixer", where)
        mixer = None
        if m:
            heads, dim = m.integer("heads", minimum=1), m.integer("dim", minimum=1)
            sizes = (heads, m.integer("kv_heads", default=heads, minimum=1), dim, m.integer("vdim", default=dim, minimum=1))
            if kind == "delta":
                mixer = DeltaConfig(*sizes, m.integer("conv", minimum=1))
            else:
                mask = section(r, m.data, "mask", where + "mixer.", required=False)
                mixer = AttentionConfig(*sizes, m.number("scale", positive=True),
                                        mask.integer("size", default=0, minimum=0) if mask else 0)
        mlp = None
        if entry.get("mlp") is not None:
            f = section(r, entry, "mlp", where)
            kindf = f.string("kind") if f else None
            if kindf == "moe":
                ex, ro = section(r, f.data, "expert", where + "mlp."), section(r, f.data, "router", where + "mlp.")
                if ex and ro:
                    mlp = MlpConfig(ex.integer("ff", minimum=1), ro.integer("experts", minimum=1), ro.integer("top", minimum=1))
            elif kindf is not None:
                r.problem(f"'{where}mlp.kind' is '{kindf}'; known: {', '.join(MLP_KINDS)}")
        return LayerConfig(kind, mixer, mlp)

    def validate(self, where="config"):
        from ..parts.recurrent import scan_fits

        problems = []
        for i, layer in enumerate(self.layers):
            if layer is None or layer.mixer is None:
                continue
            m = layer.mixer
            if m.heads % m.kv_heads:
                problems.append(f"layers[{i}]: {m.heads} heads over {m.kv_heads} kv_heads")
            if layer.type == "delta":
                if not scan_fits(m.dim, m.vdim):
                    problems.append(f"layers[{i}]: delta heads of {m.dim} key channels: the scan kernel takes up to 1024")
                if m.taps > limits.MAX_CONV_TAPS:
                    problems.append(f"layers[{i}]: {m.taps} taps: the kernels take up to {limits.MAX_CONV_TAPS}")
            elif -(-max(m.dim, m.vdim) // 16) * 16 > limits.MAX_HEAD_DIM:
                problems.append(f"layers[{i}]: attention heads of {max(m.dim, m.vdim)}: the kernels take up to {limits.MAX_HEAD_DIM}")
            if layer.mlp is not None:
                if layer.mlp.top > layer.mlp.experts:
                    problems.append(f"layers[{i}]: top {layer.mlp.top} of {layer.mlp.experts} experts")
                if layer.mlp.experts > 4096:
                    problems.append(f"layers[{i}]: {layer.mlp.experts} experts: the router kernel takes up to 4096")
        if self.streams > MAX_STREAMS:
            problems.append(f"{self.streams} streams: the kernels take up to {MAX_STREAMS}")
        if self.loop is not None and not 0 <= self.loop.start < self.loop.stop <= len(self.layers):
            problems.append(f"loop {self.loop.start}..{self.loop.stop} does not lie within {len(self.layers)} layers")
        if problems:
            raise ConfigError(f"{where}: " + "; ".join(problems))

    def with_tensor_shapes(self, shapes):
        """The same configuration, with a note of the second norm and stream factors that a checkpoint keeps for layers
        without feed-forward (nothing reads them, but they are no surprise)."""
        unused = tuple((n, tuple(shapes[n])) for i, layer in enumerate(self.layers) if layer.mlp is None
                       for n in (f"l{i}.norm2", f"l{i}.hc2.in", f"l{i}.hc2.out", f"l{i}.hc2.mix") if n in shapes)
        return dataclasses.replace(self, unused=unused)

    def run_order(self):
        """Layer indices in the order they run."""
        L = list(range(len(self.layers)))
        if self.loop is None:
            return L
        return L[:self.loop.start] + L[self.loop.start:self.loop.stop] * self.loop.times + L[self.loop.stop:]

    def to_dict(self):
        return self.raw
