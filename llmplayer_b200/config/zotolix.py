"""Configuration of the ``Zotolix`` decoder: attention in chunks of the sequence on a bundle of residual streams
(hyper-connections), values blended with an earlier layer's, and mixtures of squared-ReLU experts.

``config.json`` holds ``architecture``, ``vocab``, ``width``, ``norm: {eps}``, ``embedding: {scale}``, ``streams``,
``residual_mult`` and ``layers``, a list of ``{"type", "mixer": {...}, "mlp": {...} or null}``; layer i's tensors start
with ``l<i>.``, the mixer's with ``l<i>.mix.``, the feed-forward's with ``l<i>.mlp.``. Every sublayer has an RMS norm in front
(``norm1`` / ``norm2``) and is connected to the ``streams`` streams by ``hc1`` / ``hc2`` (``.in``, ``.out``, ``.mix``; see
``BundleBlock`` in ``parts/block.py``); ``residual_mult`` multiplies what a sublayer adds.

* both mixer types: ``heads``, ``kv_heads``, ``dim`` (queries and keys), ``vdim`` (values), ``scale``, ``mask: {size}``
  (attention inside chunks of ``size`` positions counted from the sequence's start; absent: every earlier token), ``rot:
  {base, dims}`` (pairs (i, i + dims/2); absent: no rotation), ``v_mix``. Projections with additive vectors. ``v_mix``: the
  first layer that has it shows its values to the later ones, each of which blends them into its own with the share
  ``vmix``.
* type ``attention``: after the rotation, queries and keys are divided by their root mean square per head.
* type ``attention_2``: head h's output is multiplied by sigmoid(``g`` x)_h.
* mlp ``{"kind": "moe", "expert": {"ff"}, "router": {"experts", "top"}}``: experts down(max(up x, 0)^2), the ``top`` largest
  sigmoid scores are chosen, and a score multiplies its expert's input.

The output is the model's norm ``final.norm`` of the streams' sum and the embedding table (without its scale).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple

from ..errors import ConfigError
from ..parts.specs import (
    AttentionSpec, BundleBlockSpec, ConnectionSpec, EmbeddingSpec, ExpertRoutingSpec, HeadSpec, MixtureSpec, ModelLayout, NormSpec,
    ScheduleEntry,
)
from .dopuvik import RotationConfig, _mask, _optional, _positive
from .ramupel import _need
from .registry import ArchitectureConfig, register_architecture


@dataclass(frozen=True)
class UnitHeadsConfig:
    """Attention whose queries and keys are divided by their root mean square per head."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: Optional[int]
    rot: RotationConfig
    v_mix: bool

    type = "attention"

    @classmethod
    def from_dict(cls, raw: dict, where: str):
        chunk, keep_first = _mask(raw, where)
        if keep_first:
            raise ConfigError(f"{where}mask.keep_first: chunks keep no first tokens")
        v_mix = raw.get("v_mix", False)
        if v_mix is not None and not isinstance(v_mix, bool):
            raise ConfigError(f"{where}v_mix must be true or false, got {v_mix!r}")
        return cls(heads=_need(raw, "heads", int, where), kv_heads=_need(raw, "kv_heads", int, where),
                   dim=_need(raw, "dim", int, where), vdim=_need(raw, "vdim", int, where),
                   scale=_need(raw, "scale", float, where), chunk=chunk,
                   rot=RotationConfig.from_dict(raw.get("rot"), where + "rot."), v_mix=bool(v_mix))

    def to_dict(self) -> dict:
        out = {"dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "scale": self.scale, "v_mix": self.v_mix,
               "vdim": self.vdim}
        if self.chunk is not None:
            out["mask"] = {"size": self.chunk}
        if self.rot.dims:
            out["rot"] = self.rot.to_dict()
        return out

    def validate(self, where: str) -> None:
        _positive(where, heads=self.heads, kv_heads=self.kv_heads, dim=self.dim, vdim=self.vdim)
        if self.heads % self.kv_heads:
            raise ConfigError(f"{where}heads {self.heads} is no multiple of kv_heads {self.kv_heads}")
        if self.dim > 256 or self.vdim > 256:
            raise ConfigError(f"{where}dim {self.dim} and vdim {self.vdim}: at most 256 are supported")
        if self.chunk is not None and self.chunk <= 0:
            raise ConfigError(f"{where}mask.size must be positive, got {self.chunk}")
        if self.rot.scaling is not None:
            raise ConfigError(f"{where}rot.scaling: this rotation is not stretched")
        self.rot.validate(where + "rot.", self.dim)

    def spec(self, p: str, width: int, eps: float, shows: bool):
        """``shows``: this is the first layer with ``v_mix``."""
        return AttentionSpec(
            hidden_size=width, num_heads=self.heads, num_kv_heads=self.kv_heads, head_dim=self.dim, scale=self.scale,
            position=self.rot.position(self.dim, "split_half"), q=p + "q", o=p + "o", k=p + "k", v=p + "v", value_dim=self.vdim,
            q_bias=p + "q.b", k_bias=p + "k.b", v_bias=p + "v.b", exact_weights=True, chunk=self.chunk, shows_values=shows,
            value_blend=p + "vmix" if self.v_mix and not shows else None, **self.head_rule(p, eps))

    def head_rule(self, p: str, eps: float) -> dict:
        return {"unit_norm_eps": eps}


@dataclass(frozen=True)
class GatedHeadsConfig(UnitHeadsConfig):
    """The same attention with a gate per head on its output instead of normed queries and keys."""
    type = "attention_2"

    def head_rule(self, p: str, eps: float) -> dict:
        return {"head_gate": p + "g"}


@dataclass(frozen=True)
class ExpertsConfig:
    ff: int
    experts: int
    top: int

    kind = "moe"

    @classmethod
    def from_dict(cls, raw: dict, where: str) -> "ExpertsConfig":
        router = _need(raw, "router", dict, where)
        return cls(ff=_need(_need(raw, "expert", dict, where), "ff", int, where + "expert."),
                   experts=_need(router, "experts", int, where + "router."), top=_need(router, "top", int, where + "router."))

    def to_dict(self) -> dict:
        return {"expert": {"ff": self.ff}, "kind": self.kind, "router": {"experts": self.experts, "top": self.top}}

    def validate(self, where: str) -> None:
        _positive(where, ff=self.ff, experts=self.experts, top=self.top)
        if self.top > self.experts:
            raise ConfigError(f"{where}router.top {self.top} of {self.experts} experts")

    def spec(self, p: str, width: int):
        return MixtureSpec(hidden_size=width, expert_size=self.ff, activation="relu2", weight_on="input", expert_prefix=p,
                           routing=ExpertRoutingSpec(num_experts=self.experts, top=self.top, groups=1, keep_groups=1,
                                                     router=p + "router", scoring="sigmoid_top"))


_MIXERS = {c.type: c for c in (UnitHeadsConfig, GatedHeadsConfig)}
_MLPS = {ExpertsConfig.kind: ExpertsConfig}


@dataclass(frozen=True)
class ZotolixLayerConfig:
    mixer: UnitHeadsConfig             # or GatedHeadsConfig
    mlp: Optional[ExpertsConfig]


@dataclass(frozen=True)
class ZotolixConfig(ArchitectureConfig):
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    residual_mult: float
    streams: int
    layers: Tuple[ZotolixLayerConfig, ...]

    architecture = "Zotolix"
    # the design sets no limit on positions; this is the engine's default context when none is asked for
    DEFAULT_CONTEXT = 131072

    # ------------------------------------------------------------------ reading
    @classmethod
    def from_dict(cls, raw: dict) -> "ZotolixConfig":
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
            layers.append(ZotolixLayerConfig(mixer, mlp))
        embedding = _optional(raw, "embedding", dict, "", {})
        cfg = cls(vocab=_need(raw, "vocab", int, ""), width=_need(raw, "width", int, ""),
                  norm_eps=_need(_need(raw, "norm", dict, ""), "eps", float, "norm."),
                  embedding_scale=_optional(embedding, "scale", float, "embedding.", 1.0),
                  residual_mult=_optional(raw, "residual_mult", float, "", 1.0), streams=_need(raw, "streams", int, ""),
                  layers=tuple(layers))
        cfg.validate()
        return cfg

    def validate(self) -> None:
        _positive("", vocab=self.vocab, width=self.width, streams=self.streams)
        if not self.norm_eps > 0:
            raise ConfigError(f"norm.eps must be positive, got {self.norm_eps}")
        if not self.layers:
            raise ConfigError("a model needs at least one layer")
        first = None
        for i, layer in enumerate(self.layers):
            layer.mixer.validate(f"layers[{i}].mixer.")
            if layer.mlp is not None:
                layer.mlp.validate(f"layers[{i}].mlp.")
            if layer.mixer.v_mix:
                sizes = (layer.mixer.kv_heads, layer.mixer.vdim)
                first = first if first is not None else sizes
                if sizes != first:
                    raise ConfigError(f"layers[{i}].mixer: {sizes[0]} value heads of {sizes[1]} cannot be blended with {first[0]} of {first[1]}")

    # ------------------------------------------------------------------ writing
    def to_dict(self) -> dict:
        return {
            "architecture": self.architecture,
            "embedding": {"scale": self.embedding_scale},
            "layers": [{"mixer": layer.mixer.to_dict(), "mlp": None if layer.mlp is None else layer.mlp.to_dict(),
                        "type": layer.mixer.type} for layer in self.layers],
            "norm": {"eps": self.norm_eps},
            "residual_mult": self.residual_mult,
            "streams": self.streams,
            "vocab": self.vocab,
            "width": self.width,
        }

    # ------------------------------------------------------------------ meaning
    def max_positions(self) -> int:
        return self.DEFAULT_CONTEXT

    def first_blend(self) -> Optional[int]:
        """The first layer with ``v_mix``: the one whose values the later ones blend in."""
        return next((i for i, layer in enumerate(self.layers) if layer.mixer.v_mix), None)

    def layout(self) -> ModelLayout:
        d, eps = self.width, self.norm_eps

        def connection(name: str) -> ConnectionSpec:
            return ConnectionSpec(gather=name + ".in", spread=name + ".out", mix=name + ".mix")
        shows = self.first_blend()
        blocks = []
        for i, layer in enumerate(self.layers):
            p = f"l{i}."
            has_ffn = layer.mlp is not None
            blocks.append(BundleBlockSpec(
                streams=self.streams, residual_scale=self.residual_mult,
                mixer_norm=NormSpec(d, eps, p + "norm1"), mixer=layer.mixer.spec(p + "mix.", d, eps, i == shows),
                mixer_connection=connection(p + "hc1"), ffn_norm=NormSpec(d, eps, p + "norm2") if has_ffn else None,
                ffn=layer.mlp.spec(p + "mlp.", d) if has_ffn else None, ffn_connection=connection(p + "hc2") if has_ffn else None))
        return ModelLayout(embedding=EmbeddingSpec(self.vocab, d, "embed", scale=self.embedding_scale), layers=tuple(blocks),
                           head=HeadSpec(self.vocab, d, norm=NormSpec(d, eps, "final.norm"), weight="embed"),
                           schedule=tuple(ScheduleEntry(i) for i in range(len(blocks))))

    def ignorable_tensors(self) -> tuple:
        # the first layer that blends values has no use for its share, nor has a layer that blends none; a layer without a
        # feed-forward has no use for the norm and the connection around one, should a file carry them
        shows = self.first_blend()
        spare = [f"l{i}.mix.vmix" for i, layer in enumerate(self.layers) if not layer.mixer.v_mix or i == shows]
        spare += [f"l{i}.{n}" for i, layer in enumerate(self.layers) if layer.mlp is None
                  for n in ("norm2", "hc2.in", "hc2.out", "hc2.mix")]
        return tuple(spare)

    def describe(self) -> str:
        lines = [f"architecture: {self.architecture}", f"  vocab = {self.vocab}", f"  width = {self.width}",
                 f"  norm.eps = {self.norm_eps}", f"  embedding.scale = {self.embedding_scale}",
                 f"  streams = {self.streams}", f"  residual_mult = {self.residual_mult}"]
        for i, layer in enumerate(self.layers):
            lines.append(f"  layer {i}: {layer.mixer.type} {layer.mixer.to_dict()}, feed-forward "
                         f"{None if layer.mlp is None else layer.mlp.to_dict()}")
        return "\n".join(lines)


register_architecture(ZotolixConfig.architecture, ZotolixConfig)
