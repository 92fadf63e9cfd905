"""Configuration of the ``Vomotar`` decoder: layers of a gated delta rule with a decay per key channel, and layers whose
mixer is softmax attention in chunks beside a retention, in an order the configuration lists; dense feed-forwards.

``config.json`` holds ``architecture``, ``vocab``, ``width``, ``norm: {eps, groups}`` and ``layers``, a list of
``{"type", "mixer": {...}, "mlp": {...} or null}``; layer i's tensors start with ``l<i>.``, the mixer's with ``l<i>.mix.``,
the feed-forward's with ``l<i>.mlp.``. Every layer is pre-norm with RMS norms in ``norm.groups`` equal parts of the width:
x += mixer(norm(x, norm1)); x += ffn(norm(x, norm2)).

* type ``channel_delta``: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``conv`` (taps): a gated delta rule whose decays come
  from a low-rank map, one per head and key channel, and whose output gate is the sigmoid of another low-rank map (see
  ``parts/delta_rule.py``).
* type ``parallel``: ``left`` (``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``mask: {size}``: attention without
  rotation inside chunks of ``size`` positions counted from the sequence's start, scores lowered by the tensors r1 ln(1 +
  r2 distance), values cached divided by their root mean square) and ``right`` (``heads``, ``dim``, ``vdim``, ``decay``: one
  constant per head, ``rot: {base, dims}`` with pairs (i, i + dims/2): see ``parts/retention.py``); each result is
  RMS-normed over the width (tensors ``left.out`` / ``right.out``) and half of each is added.
* mlp ``{"kind": "dense", "ff"}``: down(silu(gate x) * (up x)).

The output is the model's norm ``final.norm`` (in parts like the others) and the matrix ``head``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple

from ..errors import ConfigError
from ..parts.specs import (
    AttentionSpec, BlockSpec, EmbeddingSpec, GatedDeltaRuleSpec, HeadSpec, MixerPairSpec, ModelLayout, NormSpec, PositionSpec,
    RetentionSpec, ScheduleEntry, SwiGLUSpec,
)
from .dopuvik import RotationConfig, _mask, _optional, _positive
from .ramupel import _need
from .registry import ArchitectureConfig, register_architecture

PAIR_SHARE = 0.5        # of each of a pair's two normed results: the design fixes it


@dataclass(frozen=True)
class ChannelDeltaConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int

    type = "channel_delta"

    @classmethod
    def from_dict(cls, raw: dict, where: str) -> "ChannelDeltaConfig":
        return cls(heads=_need(raw, "heads", int, where), kv_heads=_need(raw, "kv_heads", int, where),
                   dim=_need(raw, "dim", int, where), vdim=_need(raw, "vdim", int, where), conv=_need(raw, "conv", int, where))

    def to_dict(self) -> dict:
        return {"conv": self.conv, "dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "vdim": self.vdim}

    def validate(self, where: str) -> None:
        _positive(where, heads=self.heads, kv_heads=self.kv_heads, dim=self.dim, vdim=self.vdim, conv=self.conv)
        if self.heads % self.kv_heads:
            raise ConfigError(f"{where}heads {self.heads} is no multiple of kv_heads {self.kv_heads}")
        if self.conv > 8:
            raise ConfigError(f"{where}conv {self.conv}: at most 8 taps are supported")
        if self.dim > 512:
            raise ConfigError(f"{where}dim {self.dim}: at most 512 key channels per head are supported")

    def spec(self, p: str, width: int, eps: float):
        return GatedDeltaRuleSpec(
            hidden_size=width, num_heads=self.heads, num_qk_heads=self.kv_heads, key_dim=self.dim, value_dim=self.vdim,
            conv_taps=self.conv, norm_eps=eps, q=p + "q", k=p + "k", v=p + "v", q_conv=p + "q.conv", k_conv=p + "k.conv",
            v_conv=p + "v.conv", strength=p + "b", decay=p + "a1", decay_up=p + "a2", a_log=p + "A_log", dt_bias=p + "dt_bias",
            gate=p + "g1", gate_up=p + "g2", gate_activation="sigmoid", out_norm=p + "norm", o=p + "o")


@dataclass(frozen=True)
class ChunkedAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: Optional[int]

    @classmethod
    def from_dict(cls, raw: dict, where: str) -> "ChunkedAttentionConfig":
        chunk, _ = _mask(raw, where)
        return cls(heads=_need(raw, "heads", int, where), kv_heads=_need(raw, "kv_heads", int, where),
                   dim=_need(raw, "dim", int, where), vdim=_need(raw, "vdim", int, where),
                   scale=_need(raw, "scale", float, where), chunk=chunk)

    def to_dict(self) -> dict:
        out = {"dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "scale": self.scale, "vdim": self.vdim}
        if self.chunk is not None:
            out["mask"] = {"size": self.chunk}
        return out

    def validate(self, where: str) -> None:
        _positive(where, heads=self.heads, kv_heads=self.kv_heads, dim=self.dim, vdim=self.vdim)
        if self.heads % self.kv_heads:
            raise ConfigError(f"{where}heads {self.heads} is no multiple of kv_heads {self.kv_heads}")
        if self.dim > 256 or self.vdim > 256:
            raise ConfigError(f"{where}dim {self.dim} and vdim {self.vdim}: at most 256 are supported")
        if self.chunk is not None and self.chunk <= 0:
            raise ConfigError(f"{where}mask.size must be positive, got {self.chunk}")

    def spec(self, p: str, width: int, eps: float):
        return AttentionSpec(
            hidden_size=width, num_heads=self.heads, num_kv_heads=self.kv_heads, head_dim=self.dim, scale=self.scale,
            position=PositionSpec(kind="none", head_dim=self.dim), q=p + "q", o=p + "o", k=p + "k", v=p + "v",
            value_dim=self.vdim, exact_weights=True, chunk=self.chunk, distance_scale=p + "r1", distance_rate=p + "r2",
            value_norm_eps=eps)


@dataclass(frozen=True)
class RetentionConfig:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]
    rot: RotationConfig

    @classmethod
    def from_dict(cls, raw: dict, where: str) -> "RetentionConfig":
        decay = _need(raw, "decay", list, where)
        if not all(isinstance(x, (int, float)) and not isinstance(x, bool) for x in decay):
            raise ConfigError(f"{where}decay must be a list of numbers")
        return cls(heads=_need(raw, "heads", int, where), dim=_need(raw, "dim", int, where),
                   vdim=_need(raw, "vdim", int, where), decay=tuple(float(x) for x in decay),
                   rot=RotationConfig.from_dict(raw.get("rot"), where + "rot."))

    def to_dict(self) -> dict:
        out = {"decay": list(self.decay), "dim": self.dim, "heads": self.heads, "vdim": self.vdim}
        if self.rot.dims:
            out["rot"] = self.rot.to_dict()
        return out

    def validate(self, where: str) -> None:
        _positive(where, heads=self.heads, dim=self.dim, vdim=self.vdim)
        if len(self.decay) != self.heads:
            raise ConfigError(f"{where}decay has {len(self.decay)} numbers for {self.heads} heads")
        if self.dim > 512:
            raise ConfigError(f"{where}dim {self.dim}: at most 512 key channels per head are supported")
        if self.rot.scaling is not None:
            raise ConfigError(f"{where}rot.scaling: this rotation is not stretched")
        self.rot.validate(where + "rot.", self.dim)

    def spec(self, p: str, width: int, eps: float):
        return RetentionSpec(
            hidden_size=width, num_heads=self.heads, key_dim=self.dim, value_dim=self.vdim, norm_eps=eps,
            position=self.rot.position(self.dim, "split_half"), decays=self.decay, q=p + "q", k=p + "k", v=p + "v",
            gate=p + "g", o=p + "o")


@dataclass(frozen=True)
class NormedPairConfig:
    left: ChunkedAttentionConfig
    right: RetentionConfig

    type = "parallel"

    @classmethod
    def from_dict(cls, raw: dict, where: str) -> "NormedPairConfig":
        return cls(left=ChunkedAttentionConfig.from_dict(_need(raw, "left", dict, where), where + "left."),
                   right=RetentionConfig.from_dict(_need(raw, "right", dict, where), where + "right."))

    def to_dict(self) -> dict:
        return {"left": self.left.to_dict(), "right": self.right.to_dict()}

    def validate(self, where: str) -> None:
        self.left.validate(where + "left.")
        self.right.validate(where + "right.")

    def spec(self, p: str, width: int, eps: float):
        return MixerPairSpec(
            left=self.left.spec(p + "left.", width, eps), right=self.right.spec(p + "right.", width, eps),
            left_scale=PAIR_SHARE, right_scale=PAIR_SHARE,
            left_norm=NormSpec(width, eps, p + "left.out"), right_norm=NormSpec(width, eps, p + "right.out"))


@dataclass(frozen=True)
class DenseConfig:
    ff: int

    kind = "dense"

    @classmethod
    def from_dict(cls, raw: dict, where: str) -> "DenseConfig":
        return cls(ff=_need(raw, "ff", int, where))

    def to_dict(self) -> dict:
        return {"ff": self.ff, "kind": self.kind}

    def validate(self, where: str) -> None:
        _positive(where, ff=self.ff)

    def spec(self, p: str, width: int):
        return SwiGLUSpec(hidden_size=width, intermediate_size=self.ff, gate=p + "gate", up=p + "up", down=p + "down")


_MIXERS = {c.type: c for c in (ChannelDeltaConfig, NormedPairConfig)}
_MLPS = {DenseConfig.kind: DenseConfig}


@dataclass(frozen=True)
class VomotarLayerConfig:
    mixer: object                      # ChannelDeltaConfig or NormedPairConfig
    mlp: Optional[DenseConfig]


@dataclass(frozen=True)
class VomotarConfig(ArchitectureConfig):
    vocab: int
    width: int
    norm_eps: float
    norm_groups: int
    layers: Tuple[VomotarLayerConfig, ...]

    architecture = "Vomotar"
    # the design sets no limit on positions; this is the engine's default context when none is asked for
    DEFAULT_CONTEXT = 131072

    # ------------------------------------------------------------------ reading
    @classmethod
    def from_dict(cls, raw: dict) -> "VomotarConfig":
        layers_raw = raw.get("layers")
        if not isinstance(layers_raw, list) or not layers_raw:
            raise ConfigError("config.json needs a non-empty list 'layers'")
        layers = []
        for i, entry in enumerate(layers_raw):
            where = f"layers[{i}]."
            kind = _need(entry, "type", str, where)
            if kind not in _MIXERS:
                raise ConfigError(f"{where}type {kind!r} is unknown; known: {', '.join(sorted(_MIXERS))}")
            mixer = _MIXERS[kind].from_dict(_need(entry, "mixer", dict, where), where + "mixer.")
            mlp_raw, mlp = entry.get("mlp"), None
            if mlp_raw is not None:
                if not isinstance(mlp_raw, dict):
                    raise ConfigError(f"{where}mlp must be an object or null")
                mlp_kind = _need(mlp_raw, "kind", str, where + "mlp.")
                if mlp_kind not in _MLPS:
                    raise ConfigError(f"{where}mlp.kind {mlp_kind!r} is unknown; known: {', '.join(sorted(_MLPS))}")
                mlp = _MLPS[mlp_kind].from_dict(mlp_raw, where + "mlp.")
            layers.append(VomotarLayerConfig(mixer, mlp))
        norm = _need(raw, "norm", dict, "")
        cfg = cls(vocab=_need(raw, "vocab", int, ""), width=_need(raw, "width", int, ""),
                  norm_eps=_need(norm, "eps", float, "norm."), norm_groups=_optional(norm, "groups", int, "norm.", 1),
                  layers=tuple(layers))
        cfg.validate()
        return cfg

    def validate(self) -> None:
        if self.vocab <= 0 or self.width <= 0:
            raise ConfigError(f"vocab {self.vocab} and width {self.width} must be positive")
        if not self.norm_eps > 0:
            raise ConfigError(f"norm.eps must be positive, got {self.norm_eps}")
        if self.norm_groups <= 0 or self.width % self.norm_groups:
            raise ConfigError(f"norm.groups {self.norm_groups} does not divide the width {self.width}")
        if not self.layers:
            raise ConfigError("a model needs at least one layer")
        for i, layer in enumerate(self.layers):
            layer.mixer.validate(f"layers[{i}].mixer.")
            if layer.mlp is not None:
                layer.mlp.validate(f"layers[{i}].mlp.")

    # ------------------------------------------------------------------ writing
    def to_dict(self) -> dict:
        return {
            "architecture": self.architecture,
            "layers": [{"mixer": layer.mixer.to_dict(), "mlp": None if layer.mlp is None else layer.mlp.to_dict(),
                        "type": layer.mixer.type} for layer in self.layers],
            "norm": {"eps": self.norm_eps, "groups": self.norm_groups},
            "vocab": self.vocab,
            "width": self.width,
        }

    # ------------------------------------------------------------------ meaning
    def max_positions(self) -> int:
        return self.DEFAULT_CONTEXT

    def layout(self) -> ModelLayout:
        d, eps = self.width, self.norm_eps

        def norm(name: str) -> NormSpec:
            return NormSpec(d, eps, name, groups=self.norm_groups)
        blocks = []
        for i, layer in enumerate(self.layers):
            p = f"l{i}."
            has_ffn = layer.mlp is not None
            blocks.append(BlockSpec(mixer_norm=norm(p + "norm1"), mixer=layer.mixer.spec(p + "mix.", d, eps),
                                    ffn_norm=norm(p + "norm2") if has_ffn else None,
                                    ffn=layer.mlp.spec(p + "mlp.", d) if has_ffn else None))
        return ModelLayout(embedding=EmbeddingSpec(self.vocab, d, "embed"), layers=tuple(blocks),
                           head=HeadSpec(self.vocab, d, norm=norm("final.norm"), weight="head"),
                           schedule=tuple(ScheduleEntry(i) for i in range(len(blocks))))

    def ignorable_tensors(self) -> tuple:
        # a layer without a feed-forward has no use for the norm in front of one, should a file carry it
        return tuple(f"l{i}.norm2" for i, layer in enumerate(self.layers) if layer.mlp is None)

    def describe(self) -> str:
        lines = [f"architecture: {self.architecture}", f"  vocab = {self.vocab}", f"  width = {self.width}",
                 f"  norm.eps = {self.norm_eps}", f"  norm.groups = {self.norm_groups}"]
        for i, layer in enumerate(self.layers):
            lines.append(f"  layer {i}: {layer.mixer.type} {layer.mixer.to_dict()}, feed-forward "
                         f"{None if layer.mlp is None else layer.mlp.to_dict()}")
        return "\n".join(lines)


register_architecture(VomotarConfig.architecture, VomotarConfig)
