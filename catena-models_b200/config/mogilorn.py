"""Configuration of the Mogilorn decoder.

config.json is nested: `vocab`, `width`, `norm.eps`, `embedding.scale` (the factor on every embedding row); `layers`,
a list whose entries give `type` (which mixer the layer has), `mixer` (its sizes and constants) and `mlp` (the
feed-forward, or null for none).

Mixer types: `attention` (`heads`, `kv_heads`, `dim`, `vdim`, `scale`, `softcap`, `rot.dims`, `rot.base`,
`rot.scaling.{factor, low, high, original}`, `v_mix`: the layer mixes its values with those of the first layer that says
so), `mlstm` (`heads`, `dim`, `vdim`, `gate_cap`) and `latent_attention` (`heads`, `dim`, `rot_dim`, `vdim`, `kv_rank`,
`scale`, `rot.dims`, `rot.base`, `rot.scaling`, `mask.size`: the sliding window).  Feed-forward kind: `dense` (`ff`).
"""
from __future__ import annotations

import dataclasses

from ..csrc import limits
from .base import ConfigError, Reader, base_type, section

MIXER_TYPES = ("attention", "mlstm", "latent_attention")
MLP_KINDS = ("dense",)


@dataclasses.dataclass(frozen=True)
class ScalingConfig:
    factor: float
    low: float
    high: float
    original: float


@dataclasses.dataclass(frozen=True)
class RotationConfig:
    dims: int
    base: float
    scaling: object          # ScalingConfig, or None: the rates are not rescaled


@dataclasses.dataclass(frozen=True)
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: float           # 0: none
    v_mix: bool
    rot: object              # RotationConfig or None


@dataclasses.dataclass(frozen=True)
class MatrixMemoryConfig:
    heads: int
    dim: int
    vdim: int
    gate_cap: float


@dataclasses.dataclass(frozen=True)
class LatentAttentionConfig:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    window: int              # 0: every earlier position is seen
    rot: object              # RotationConfig or None


@dataclasses.dataclass(frozen=True)
class MlpConfig:
    ff: int


@dataclasses.dataclass(frozen=True)
class LayerConfig:
    type: str
    mixer: object
    mlp: object              # MlpConfig or None


def _rotation(r, m, where):
    rot = section(r, m.data, "rot", where + "mixer.", required=False)
    if not rot:
        return None
    sc = section(r, rot.data, "scaling", where + "mixer.rot.", required=False)
    scaling = ScalingConfig(*(sc.number(k, positive=True) for k in ("factor", "low", "high", "original"))) if sc else None
    return RotationConfig(rot.integer("dims", minimum=2), rot.number("base", positive=True), scaling)


@dataclasses.dataclass(frozen=True)
class MogilornConfig:
    architecture: str
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    layers: tuple
    unused: tuple = ()       # (name, shape) of tensors that a checkpoint carries although no part reads them
    raw: dict = dataclasses.field(compare=False, default=None)

    @classmethod
    def from_dict(cls, data, where="config.json"):
        r = Reader(data, where)
        arch = r.string("architecture")
        vocab, width = r.integer("vocab", minimum=1), r.integer("width", minimum=1)
        norm = section(r, data, "norm", "")
        eps = norm.number("eps", positive=True) if norm else None
        emb = section(r, data, "embedding", "", required=False)
        emb_scale = emb.number("scale", default=1.0) if emb else 1.0
        raw_layers = data.get("layers")
        if not isinstance(raw_layers, list) or not raw_layers:
            r.problem("'layers' must be a non-empty list")
            raw_layers = []
        layers = [cls._layer(r, entry, f"layers[{i}].") for i, entry in enumerate(raw_layers)]
        r.finish()
        cfg = cls(arch, vocab, width, eps, emb_scale, tuple(layers), raw=data)
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
            vdim = m.integer("vdim", default=dim, minimum=1)
            if kind == "attention":
                mixer = AttentionConfig(heads, m.integer("kv_heads", default=heads, minimum=1), dim, vdim,
                                        m.number("scale", positive=True), m.number("softcap", default=0.0),
                                        m.boolean("v_mix", default=False), _rotation(r, m, where))
            elif kind == "mlstm":
                mixer = MatrixMemoryConfig(heads, dim, vdim, m.number("gate_cap", positive=True))
            else:
                mask = section(r, m.data, "mask", where + "mixer.", required=False)
                mixer = LatentAttentionConfig(heads, dim, m.integer("rot_dim", default=0, minimum=0), vdim,
                                              m.integer("kv_rank", minimum=1), m.number("scale", positive=True),
                                              mask.integer("size", default=0, minimum=0) if mask else 0, _rotation(r, m, where))
        mlp = None
        if entry.get("mlp") is not None:
            f = section(r, entry, "mlp", where)
            kindf = f.string("kind") if f else None
            if kindf == "dense":
                mlp = MlpConfig(f.integer("ff", minimum=1))
            elif kindf is not None:
                r.problem(f"'{where}mlp.kind' is '{kindf}'; known: {', '.join(MLP_KINDS)}")
        return LayerConfig(kind, mixer, mlp)

    def value_source(self):
        """The layer whose values the others mix in (the first that says `v_mix`), or None."""
        return next((i for i, layer in enumerate(self.layers) if layer.type == "attention" and layer.mixer.v_mix), None)

    def validate(self, where="config"):
        from ..parts.recurrent import scan_fits

        problems = []
        for i, layer in enumerate(self.layers):
            m = layer.mixer
            rot, turned = getattr(m, "rot", None), m.rot_dim if layer.type == "latent_attention" else m.dim
            if rot is not None and (rot.dims % 2 or rot.dims > turned):
                problems.append(f"layers[{i}]: {rot.dims} turned channels in a part of {turned}")
            if rot is not None and rot.scaling is not None and rot.scaling.high <= rot.scaling.low:
                problems.append(f"layers[{i}]: rotation scaling with high {rot.scaling.high} not above low {rot.scaling.low}")
            if layer.type == "attention":
                if m.heads % m.kv_heads:
                    problems.append(f"layers[{i}]: {m.heads} heads over {m.kv_heads} kv_heads")
                if -(-max(m.dim, m.vdim) // 16) * 16 > limits.MAX_HEAD_DIM:
                    problems.append(f"layers[{i}]: attention heads of {max(m.dim, m.vdim)}: the kernels take up to {limits.MAX_HEAD_DIM}")
                if m.softcap < 0.0:
                    problems.append(f"layers[{i}]: a softcap of {m.softcap}")
                src = self.layers[self.value_source()].mixer if m.v_mix else m
                if src.kv_heads * src.vdim != m.kv_heads * m.vdim:
                    problems.append(f"layers[{i}]: mixes {m.kv_heads * m.vdim} value channels with {src.kv_heads * src.vdim}")
            elif layer.type == "mlstm":
                if not scan_fits(m.dim, m.vdim):
                    problems.append(f"layers[{i}]: matrix-memory heads of {m.dim} key channels: the scan kernel takes up to 1024")
            elif m.kv_rank > 512:
                problems.append(f"layers[{i}]: latents of {m.kv_rank} channels: the kernels take up to 512")
        if problems:
            raise ConfigError(f"{where}: " + "; ".join(problems))

    def with_tensor_shapes(self, shapes):
        """The same configuration, with a note of tensors that a checkpoint may keep for layers that do not read them: the
        second norm of a layer without feed-forward, the share of a layer that mixes no values."""
        unused = []
        for i, layer in enumerate(self.layers):
            names = [f"l{i}.norm2"] if layer.mlp is None else []
            if layer.type == "attention" and not layer.mixer.v_mix:
                names.append(f"l{i}.mix.vmix")
            unused += [(n, tuple(shapes[n])) for n in names if n in shapes]
        return dataclasses.replace(self, unused=tuple(unused))

    def to_dict(self):
        return self.raw
