"""Mugulorn: its typed configuration and the architecture entry.

A decoder with a norm in front of every sublayer and one constant that multiplies what every
sublayer adds to the stream:

    x <- x + m mixer(norm1(x));   x <- x + m ff(norm2(x))        (the second half where the layer has a feed-forward)

A layer's mixer is one of two.  "latent_attention": attention inside a sliding window whose queries pass
a normed latent and whose keys and values are rebuilt from a normed latent c plus one rotated key part
for all heads (entry i turns with entry i + half; frequencies stretched by a ramp between two
wavelengths, cosines and sines times 0.1 ln(factor) + 1), with a learned score per head in the softmax's
denominator and the heads' outputs multiplied by the sigmoid of a projection of the mixer's input; only
[c ; rotated part] is cached, and a layer may read the rows another layer cached (`kv_from`) with
matrices, window and sinks of its own.  "rglru": two branches, gelu(W_y h + b) and a short convolution of
W_x h + b, the second through a recurrence per channel whose decay and input gate come from products of
that branch in diagonal blocks.  The feed-forward is W_down (gelu(W_gate h) * (W_up h)) with the tanh form
of gelu.  The embedding rows carry a multiplier; the table without it is the output matrix.  Every size
and every constant that may differ between two models of the design comes from config.json:

    architecture, vocab, width, norm.eps, embedding.scale, residual_mult
    layers[i] {type, mixer {...}, mlp null | {kind: "dense", ff}}
      type "latent_attention": mixer {heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, mask {size},
                                      rot {base, dims, scaling {factor, original, fast, slow} (optional)}, kv_from (optional)}
      type "rglru":            mixer {width, blocks, conv}

Tensor names: embed, l<i>.norm1/.norm2, l<i>.mix.{dq,dq.norm,uq,dkv,dkv.norm,uk,uv,sink,g,o},
l<i>.mix.{y,y.b,x,x.b,conv,conv.b,ra,ra.b,ri,ri.b,lam,o}, l<i>.mlp.{gate,up,down}, final.norm.
Constants in code are those the design fixes: 8 in the decay's exponent, 0.1 ln(factor) + 1 and 0.001 in
the stretched rotation.
"""

from __future__ import annotations

from dataclasses import dataclass, field, replace
from pathlib import Path
from typing import Any, Optional, Union

from tokensprint_b200.config.model_config import ConfigError, read_config_json, require, write_config_json
from tokensprint_b200.config.registry import PRESET_DIR, register_architecture, register_preset
from tokensprint_b200.models.spec import ModelSpec, RunSpec
from tokensprint_b200.models.vasosun import LatentAttentionConfig, _section
from tokensprint_b200.parts.base import PartSpec

ARCHITECTURE = "Mugulorn"
DEFAULT_MAX_POSITIONS = 32768  # the design sets no limit; what the engine plans for unless the file says otherwise
DECAY_SCALE = 8.0


@dataclass(frozen=True)
class WindowLatentConfig(LatentAttentionConfig):
    """A latent attention inside a sliding window, with sinks and an output gate."""

    window: int = 0  # 0: every earlier key

    @classmethod
    def from_dict(cls, d: dict[str, Any], where: str) -> "WindowLatentConfig":
        window = require(_section(d, "mask", where), "size", int) if d.get("mask") is not None else 0
        if d.get("mask") is not None and window < 1:
            raise ConfigError(f"config.json: {where}mask.size must be positive")
        return replace(super().from_dict(d, where), window=window)

    def to_dict(self) -> dict[str, Any]:
        d = super().to_dict()
        if self.window:
            d["mask"] = {"size": self.window}
        return d

    def part(self, width: int, eps: float, p: str) -> PartSpec:
        base = super().part(width, eps, p)
        params = dict(base.params, window=self.window, sink=p + "sink", out_gate=p + "g")
        if params["position"] is not None:
            params["position"] = PartSpec("rotary", dict(params["position"].params, pairing="half"))
        return PartSpec(base.kind, params)


@dataclass(frozen=True)
class RecurrentConfig:
    width: int
    blocks: int
    conv: int

    @classmethod
    def from_dict(cls, d: dict[str, Any], where: str) -> "RecurrentConfig":
        c = cls(*(require(d, k, int) for k in ("width", "blocks", "conv")))
        if min(c.width, c.blocks, c.conv) < 1 or c.width % c.blocks:
            raise ConfigError(f"config.json: {where}sizes must be positive and width a multiple of blocks")
        return c

    def to_dict(self) -> dict[str, Any]:
        return {"width": self.width, "blocks": self.blocks, "conv": self.conv}

    def part(self, width: int, eps: float, p: str) -> PartSpec:
        return PartSpec("gated_recurrence", {
            "hidden_size": width, "width": self.width, "blocks": self.blocks, "taps": self.conv, "decay_scale": DECAY_SCALE,
            "y": p + "y", "y_bias": p + "y.b", "x": p + "x", "x_bias": p + "x.b", "conv": p + "conv", "conv_bias": p + "conv.b",
            "r": p + "ra", "r_bias": p + "ra.b", "i": p + "ri", "i_bias": p + "ri.b", "lam": p + "lam", "o": p + "o"})


MIXER_CONFIGS = {"latent_attention": WindowLatentConfig, "rglru": RecurrentConfig}
MixerConfig = Union[WindowLatentConfig, RecurrentConfig]


@dataclass(frozen=True)
class MugulornLayerConfig:
    type: str
    mixer: MixerConfig
    ff: int = 0  # inner width of the feed-forward; 0: none


@dataclass(frozen=True)
class MugulornConfig:
    """All sizes and constants of one Mugulorn model."""

    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    residual_mult: float
    layers: tuple[MugulornLayerConfig, ...]
    max_position_embeddings: int = DEFAULT_MAX_POSITIONS
    eos_token_id: int = -1
    extra: dict[str, Any] = field(default_factory=dict, compare=False, repr=False)

    def __post_init__(self) -> None:
        if self.vocab < 1 or self.width < 1 or not self.layers:
            raise ConfigError("config.json: 'vocab', 'width' and the number of layers must be positive")
        if self.norm_eps <= 0:
            raise ConfigError("config.json: 'norm.eps' must be positive")
        for i, layer in enumerate(self.layers):
            m = layer.mixer
            if isinstance(m, WindowLatentConfig) and m.kv_from is not None:
                j = m.kv_from
                source = self.layers[j].mixer if 0 <= j < i else None
                if not isinstance(source, WindowLatentConfig) or source.kv_from is not None or not m.cached_like(source):
                    raise ConfigError(f"config.json: layers[{i}].mixer.kv_from must name an earlier latent attention layer with a latent "
                                      f"of its own and the same kv_rank, rot_dim and rotation")

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    @classmethod
    def from_dict(cls, d: dict[str, Any]) -> "MugulornConfig":
        entries = d.get("layers")
        if not isinstance(entries, list) or not entries:
            raise ConfigError("config.json: 'layers' must be a list with an entry per layer")
        layers = []
        for i, entry in enumerate(entries):
            where = f"layers[{i}]."
            kind = entry.get("type")
            if kind not in MIXER_CONFIGS:
                raise ConfigError(f"config.json: {where}type {kind!r} is no mixer of this design (known: {sorted(MIXER_CONFIGS)})")
            mlp, ff = entry.get("mlp"), 0
            if mlp is not None:
                if mlp.get("kind") != "dense":
                    raise ConfigError(f"config.json: {where}mlp.kind must be 'dense', got {mlp.get('kind')!r}")
                ff = require(mlp, "ff", int)
                if ff < 1:
                    raise ConfigError(f"config.json: {where}mlp.ff must be positive")
            layers.append(MugulornLayerConfig(type=kind, mixer=MIXER_CONFIGS[kind].from_dict(_section(entry, "mixer", where), where), ff=ff))
        known = {"architecture", "architectures", "model_type", "vocab", "width", "norm", "layers", "embedding", "residual_mult",
                 "max_position_embeddings", "eos_token_id"}
        return cls(
            vocab=require(d, "vocab", int), width=require(d, "width", int), norm_eps=require(_section(d, "norm", ""), "eps", float),
            embedding_scale=require(_section(d, "embedding", ""), "scale", float), residual_mult=require(d, "residual_mult", float),
            layers=tuple(layers), max_position_embeddings=int(d.get("max_position_embeddings") or DEFAULT_MAX_POSITIONS),
            eos_token_id=int(d["eos_token_id"]) if isinstance(d.get("eos_token_id"), int) else -1,
            extra={k: v for k, v in d.items() if k not in known})

    @classmethod
    def from_json(cls, path: str | Path) -> "MugulornConfig":
        return cls.from_dict(read_config_json(path))

    def to_dict(self) -> dict[str, Any]:
        layers = [{"type": l.type, "mixer": l.mixer.to_dict(), "mlp": {"kind": "dense", "ff": l.ff} if l.ff else None} for l in self.layers]
        d: dict[str, Any] = {"architecture": ARCHITECTURE, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
                             "embedding": {"scale": self.embedding_scale}, "residual_mult": self.residual_mult, "layers": layers}
        if self.max_position_embeddings != DEFAULT_MAX_POSITIONS:
            d["max_position_embeddings"] = self.max_position_embeddings
        if self.eos_token_id >= 0:
            d["eos_token_id"] = self.eos_token_id
        return d

    def save(self, folder: str | Path) -> None:
        write_config_json(folder, self.to_dict())


@register_architecture(ARCHITECTURE, model_types=("mugulorn",), config_from_dict=MugulornConfig.from_dict)
def build_mugulorn_spec(config: MugulornConfig) -> ModelSpec:
    W, eps = config.width, config.norm_eps

    def norm(name: str) -> PartSpec:
        return PartSpec("rmsnorm", {"dim": W, "eps": eps, "weight": name})

    blocks: list[PartSpec] = []
    runs: list[RunSpec] = []
    ignorable: list[str] = []
    sources = {i: l.mixer.kv_from for i, l in enumerate(config.layers) if isinstance(l.mixer, WindowLatentConfig) and l.mixer.kv_from is not None}
    for i, layer in enumerate(config.layers):
        p = f"l{i}."
        params: dict[str, Any] = {"mixer": layer.mixer.part(W, eps, p + "mix."), "mixer_norm": norm(p + "norm1"),
                                  "residual_scale": config.residual_mult}
        if layer.ff:
            params.update(ffn_norm=norm(p + "norm2"), feed_forward=PartSpec("swiglu", {
                "hidden_size": W, "intermediate_size": layer.ff, "gate": p + "mlp.gate", "up": p + "mlp.up", "down": p + "mlp.down",
                "activation": "gelu_tanh"}))
        else:
            ignorable.append(p + "norm2")  # a layer without a feed-forward has no use for it
        blocks.append(PartSpec("pre_norm", params))
        # a layer that reads another layer's cached rows is a run that shares that layer's cache without writing it
        if i in sources:
            runs.append(RunSpec(layer=i, cache=sources[i], writes_cache=False))
        else:
            runs.append(RunSpec(layer=i, cache=i if i in sources.values() else None))
    return ModelSpec(vocab_size=config.vocab, hidden_size=W, embedding="embed", layers=blocks, final_norm=norm("final.norm"), lm_head=None,
                     run_order=runs, max_positions=config.max_position_embeddings, eos_token_id=config.eos_token_id,
                     ignorable_tensors=tuple(ignorable), embedding_scale=config.embedding_scale)


# Named models of this design, so that the command lines can run them with random weights.
for _path in sorted(PRESET_DIR.glob("mugulorn-*.json")):
    register_preset("mugulorn", _path.stem, _path)
