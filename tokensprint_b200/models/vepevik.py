"""Vepevik: its typed configuration and the architecture entry.

A pre-norm decoder over a normed embedding, x = N_embed(embed[token]), with logits from the embedding
table itself.  A layer's mixer is one of three.  "attention": grouped-query softmax attention that
sees only the keys of its own chunk of positions, with a weighted norm per q and k head before a
rotation of the first entries, values that may differ in width from keys, a sigmoid gate per head, and
(`v_mix`) values blended with those that the first such layer made for the same token.  "retention":
a linear recurrence over rotated q and k with one constant decay per head, each head's read-out
divided by its root mean square, a silu gate.  "channel_delta": the gated delta rule with a decay per
head and key channel; decay and sigmoid output gate pass narrow pairs of matrices.  The feed-forward
is dense with capped operands or a set of routed SwiGLU experts: softmax scores, a choice inside the
best groups of experts, weights divided by their sum and multiplied by a constant.  Every size and
every constant that may differ between two models of the design comes from config.json:

    architecture, vocab, width, norm.eps
    layers[i] {type, mixer {...}, mlp null | {kind: "dense", ff, limit}
                                           | {kind: "moe", expert {ff}, router {experts, top, scale, groups {count, keep} (optional)}}}
      type "attention":      mixer {heads, kv_heads, dim, vdim, scale, rot {base, dims} (optional), mask {size} (optional), v_mix (optional)}
      type "retention":      mixer {heads, dim, vdim, decay [heads], rot {base, dims} (optional)}
      type "channel_delta":  mixer {heads, kv_heads, dim, vdim, conv, decay_rank, gate_rank (optional: else the tensors' own)}

Tensor names: embed, embed.norm, l<i>.norm1/.norm2, l<i>.mix.{q,k,v,q.norm,k.norm,g,vmix,o},
l<i>.mix.{q,k,v,g,o}, l<i>.mix.{q,q.conv,k,k.conv,v,v.conv,b,A_log,a1,a2,dt_bias,norm,g1,g2,o},
l<i>.mlp.{gate,up,down}, l<i>.mlp.{router,e<j>.{gate,up,down}}, final.norm.
Constants in code are those the design fixes: 1e-6 under the unit length of q and k and the key width's
inverse root on q (delta rule) or k (retention), 1.702 in the capped feed-forward.
"""

from __future__ import annotations

from dataclasses import dataclass, field
from pathlib import Path
from typing import Any, Optional, Union

from tokensprint_b200.config.model_config import ConfigError, read_config_json, require, write_config_json
from tokensprint_b200.config.registry import PRESET_DIR, register_architecture, register_preset
from tokensprint_b200.models.spec import ModelSpec
from tokensprint_b200.parts.base import PartSpec

ARCHITECTURE = "Vepevik"
DEFAULT_MAX_POSITIONS = 32768  # the design sets no limit; what the engine plans for unless the file says otherwise
FIRST_VALUES = "first"         # under which the first blending layer leaves its values in a step


def _section(d: dict[str, Any], key: str, where: str) -> dict[str, Any]:
    value = d.get(key)
    if not isinstance(value, dict):
        raise ConfigError(f"config.json: {where}'{key}' must be an object")
    return value


@dataclass(frozen=True)
class RotationConfig:
    base: float
    dims: int  # entries at the front of a head that turn

    @classmethod
    def from_dict(cls, d: dict[str, Any], dim: int, where: str) -> Optional["RotationConfig"]:
        if d.get("rot") is None:
            return None
        rot = _section(d, "rot", where)
        c = cls(require(rot, "base", float), require(rot, "dims", int))
        if c.dims % 2 or not 0 <= c.dims <= dim or c.base <= 0:
            raise ConfigError(f"config.json: {where}rot.dims must be even and at most dim, rot.base positive")
        return c

    def to_dict(self) -> dict[str, Any]:
        return {"base": self.base, "dims": self.dims}

    def part(self) -> Optional[PartSpec]:
        return PartSpec("rotary", {"dim": self.dims, "theta": self.base, "exact_frequencies": True}) if self.dims else None


@dataclass(frozen=True)
class ChunkAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Optional[RotationConfig]
    chunk: int    # 0: every earlier key
    v_mix: bool

    @classmethod
    def from_dict(cls, d: dict[str, Any], where: str) -> "ChunkAttentionConfig":
        heads, kv_heads, dim, vdim = (require(d, k, int) for k in ("heads", "kv_heads", "dim", "vdim"))
        if min(heads, kv_heads, dim, vdim) < 1 or heads % kv_heads:
            raise ConfigError(f"config.json: {where}heads must be a positive multiple of kv_heads, dim and vdim positive")
        chunk = require(_section(d, "mask", where), "size", int) if d.get("mask") is not None else 0
        if chunk < 0 or (d.get("mask") is not None and chunk < 1):
            raise ConfigError(f"config.json: {where}mask.size must be positive")
        return cls(heads, kv_heads, dim, vdim, require(d, "scale", float), RotationConfig.from_dict(d, dim, where), chunk, bool(d.get("v_mix", False)))

    def to_dict(self) -> dict[str, Any]:
        d: dict[str, Any] = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale}
        if self.rot is not None:
            d["rot"] = self.rot.to_dict()
        if self.chunk:
            d["mask"] = {"size": self.chunk}
        if self.v_mix:
            d["v_mix"] = True
        return d

    def part(self, width: int, eps: float, p: str, leads: bool) -> PartSpec:
        """`leads`: the first layer that blends, whose values the others take in."""
        return PartSpec("attention", {
            "hidden_size": width, "num_heads": self.heads, "num_kv_heads": self.kv_heads, "head_dim": self.dim, "value_dim": self.vdim,
            "scale": self.scale, "chunk": self.chunk, "qk_norm": "head", "qk_norm_eps": eps, "q_norm": p + "q.norm", "k_norm": p + "k.norm",
            "position": self.rot.part() if self.rot is not None else None, "gate": p + "g", "gate_per": "head",
            "shares_values": FIRST_VALUES if leads else None,
            "value_mix": (FIRST_VALUES, p + "vmix") if self.v_mix and not leads else None,
            "q": p + "q", "k": p + "k", "v": p + "v", "o": p + "o"})


@dataclass(frozen=True)
class RetentionConfig:
    heads: int
    dim: int
    vdim: int
    decay: tuple[float, ...]
    rot: Optional[RotationConfig]

    @classmethod
    def from_dict(cls, d: dict[str, Any], where: str) -> "RetentionConfig":
        heads, dim, vdim = (require(d, k, int) for k in ("heads", "dim", "vdim"))
        decay = d.get("decay")
        if min(heads, dim, vdim) < 1:
            raise ConfigError(f"config.json: {where}heads, dim and vdim must be positive")
        if not isinstance(decay, list) or len(decay) != heads or not all(isinstance(a, (int, float)) and not isinstance(a, bool) for a in decay):
            raise ConfigError(f"config.json: {where}decay must list one number per head")
        return cls(heads, dim, vdim, tuple(float(a) for a in decay), RotationConfig.from_dict(d, dim, where))

    def to_dict(self) -> dict[str, Any]:
        d: dict[str, Any] = {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "decay": list(self.decay)}
        if self.rot is not None:
            d["rot"] = self.rot.to_dict()
        return d

    def part(self, width: int, eps: float, p: str) -> PartSpec:
        return PartSpec("retention", {
            "hidden_size": width, "num_heads": self.heads, "key_dim": self.dim, "value_dim": self.vdim, "decay": self.decay, "norm_eps": eps,
            "position": self.rot.part() if self.rot is not None else None, "q": p + "q", "k": p + "k", "v": p + "v", "gate": p + "g", "o": p + "o"})


@dataclass(frozen=True)
class ChannelDeltaConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    decay_rank: Optional[int] = None  # None: the inner widths are read from the tensors
    gate_rank: Optional[int] = None

    @classmethod
    def from_dict(cls, d: dict[str, Any], where: str) -> "ChannelDeltaConfig":
        ranks = [require(d, k, int) if d.get(k) is not None else None for k in ("decay_rank", "gate_rank")]
        c = cls(*(require(d, k, int) for k in ("heads", "kv_heads", "dim", "vdim", "conv")), *ranks)
        if min(c.heads, c.kv_heads, c.dim, c.vdim, c.conv) < 1 or c.heads % c.kv_heads or any(r is not None and r < 1 for r in ranks):
            raise ConfigError(f"config.json: {where}sizes must be positive and heads a multiple of kv_heads")
        return c

    def to_dict(self) -> dict[str, Any]:
        d: dict[str, Any] = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "conv": self.conv}
        for key in ("decay_rank", "gate_rank"):
            if getattr(self, key) is not None:
                d[key] = getattr(self, key)
        return d

    def part(self, width: int, eps: float, p: str) -> PartSpec:
        return PartSpec("gated_delta_rule", {
            "hidden_size": width, "num_heads": self.heads, "num_qk_heads": self.kv_heads, "key_dim": self.dim, "value_dim": self.vdim,
            "taps": self.conv, "norm_eps": eps, "unit_eps": 1e-6, "q": p + "q", "k": p + "k", "v": p + "v", "q_conv": p + "q.conv",
            "k_conv": p + "k.conv", "v_conv": p + "v.conv", "beta": p + "b", "a_log": p + "A_log", "dt_bias": p + "dt_bias",
            "decay_pair": (p + "a1", p + "a2"), "gate_pair": (p + "g1", p + "g2"), "decay_rank": self.decay_rank, "gate_rank": self.gate_rank,
            "gate_activation": "sigmoid", "norm": p + "norm", "o": p + "o"})


@dataclass(frozen=True)
class DenseConfig:
    ff: int
    limit: float

    @classmethod
    def from_dict(cls, d: dict[str, Any], where: str) -> "DenseConfig":
        c = cls(require(d, "ff", int), require(d, "limit", float))
        if c.ff < 1:
            raise ConfigError(f"config.json: {where}mlp.ff must be positive")
        return c

    def to_dict(self) -> dict[str, Any]:
        return {"kind": "dense", "ff": self.ff, "limit": self.limit}

    def part(self, width: int, p: str) -> PartSpec:
        return PartSpec("capped_glu", {"hidden_size": width, "intermediate_size": self.ff, "limit": self.limit, "alpha": 1.702,
                                       "gate": p + "gate", "up": p + "up", "down": p + "down"})


@dataclass(frozen=True)
class ExpertsConfig:
    ff: int
    experts: int
    top: int
    scale: float
    groups: Optional[tuple[int, int]]  # (count, keep), or None: no groups

    @classmethod
    def from_dict(cls, d: dict[str, Any], where: str) -> "ExpertsConfig":
        where += "mlp."
        router = _section(d, "router", where)
        groups = None
        if router.get("groups") is not None:
            g = _section(router, "groups", where + "router.")
            groups = (require(g, "count", int), require(g, "keep", int))
        c = cls(require(_section(d, "expert", where), "ff", int), require(router, "experts", int), require(router, "top", int),
                require(router, "scale", float) if router.get("scale") is not None else 1.0, groups)
        if c.ff < 1 or not 0 < c.top <= c.experts:
            raise ConfigError(f"config.json: {where}router.top must lie in 1..router.experts, expert.ff be positive")
        if groups is not None:
            count, keep = groups
            if count < 1 or c.experts % count or not 1 <= keep <= count or c.top > keep * (c.experts // count):
                raise ConfigError(f"config.json: {where}router.groups: count must divide experts, keep lie in 1..count and leave `top` experts")
        return c

    def to_dict(self) -> dict[str, Any]:
        router: dict[str, Any] = {"experts": self.experts, "top": self.top, "scale": self.scale}
        if self.groups is not None:
            router["groups"] = {"count": self.groups[0], "keep": self.groups[1]}
        return {"kind": "moe", "expert": {"ff": self.ff}, "router": router}

    def part(self, width: int, p: str) -> PartSpec:
        return PartSpec("routed_experts", {
            "hidden_size": width, "num_experts": self.experts, "top": self.top, "intermediate_size": self.ff, "router": p + "router",
            "expert_prefix": p + "e", "score": "softmax_all", "renormalize": True, "weight_scale": self.scale, "groups": self.groups,
            "activation": "swiglu", "weight_on": "output"})


MIXER_CONFIGS = {"attention": ChunkAttentionConfig, "retention": RetentionConfig, "channel_delta": ChannelDeltaConfig}
FEED_FORWARD_CONFIGS = {"dense": DenseConfig, "moe": ExpertsConfig}


@dataclass(frozen=True)
class VepevikLayerConfig:
    type: str
    mixer: Union[ChunkAttentionConfig, RetentionConfig, ChannelDeltaConfig]
    mlp: Optional[Union[DenseConfig, ExpertsConfig]] = None


@dataclass(frozen=True)
class VepevikConfig:
    """All sizes and constants of one Vepevik model."""

    vocab: int
    width: int
    norm_eps: float
    layers: tuple[VepevikLayerConfig, ...]
    max_position_embeddings: int = DEFAULT_MAX_POSITIONS
    eos_token_id: int = -1
    extra: dict[str, Any] = field(default_factory=dict, compare=False, repr=False)

    def __post_init__(self) -> None:
        if self.vocab < 1 or self.width < 1 or not self.layers:
            raise ConfigError("config.json: 'vocab', 'width' and the number of layers must be positive")
        if self.norm_eps <= 0:
            raise ConfigError("config.json: 'norm.eps' must be positive")
        blending = [self.layers[i].mixer for i in self.blending_layers]
        if any((m.kv_heads, m.vdim) != (blending[0].kv_heads, blending[0].vdim) for m in blending):
            raise ConfigError("config.json: layers with v_mix blend their values and so need the same kv_heads and vdim")

    @property
    def blending_layers(self) -> list[int]:
        return [i for i, l in enumerate(self.layers) if isinstance(l.mixer, ChunkAttentionConfig) and l.mixer.v_mix]

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    @classmethod
    def from_dict(cls, d: dict[str, Any]) -> "VepevikConfig":
        entries = d.get("layers")
        if not isinstance(entries, list) or not entries:
            raise ConfigError("config.json: 'layers' must be a list with an entry per layer")
        layers = []
        for i, entry in enumerate(entries):
            where = f"layers[{i}]."
            kind, mlp = entry.get("type"), entry.get("mlp")
            if kind not in MIXER_CONFIGS:
                raise ConfigError(f"config.json: {where}type {kind!r} is no mixer of this design (known: {sorted(MIXER_CONFIGS)})")
            if mlp is not None and mlp.get("kind") not in FEED_FORWARD_CONFIGS:
                raise ConfigError(f"config.json: {where}mlp.kind must be one of {sorted(FEED_FORWARD_CONFIGS)}, got {mlp.get('kind')!r}")
            layers.append(VepevikLayerConfig(type=kind, mixer=MIXER_CONFIGS[kind].from_dict(_section(entry, "mixer", where), where),
                                             mlp=None if mlp is None else FEED_FORWARD_CONFIGS[mlp["kind"]].from_dict(mlp, where)))
        known = {"architecture", "architectures", "model_type", "vocab", "width", "norm", "layers", "max_position_embeddings", "eos_token_id"}
        return cls(vocab=require(d, "vocab", int), width=require(d, "width", int), norm_eps=require(_section(d, "norm", ""), "eps", float),
                   layers=tuple(layers), max_position_embeddings=int(d.get("max_position_embeddings") or DEFAULT_MAX_POSITIONS),
                   eos_token_id=int(d["eos_token_id"]) if isinstance(d.get("eos_token_id"), int) else -1,
                   extra={k: v for k, v in d.items() if k not in known})

    @classmethod
    def from_json(cls, path: str | Path) -> "VepevikConfig":
        return cls.from_dict(read_config_json(path))

    def to_dict(self) -> dict[str, Any]:
        layers = [{"type": l.type, "mixer": l.mixer.to_dict(), "mlp": None if l.mlp is None else l.mlp.to_dict()} for l in self.layers]
        d: dict[str, Any] = {"architecture": ARCHITECTURE, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
                             "layers": layers}
        if self.max_position_embeddings != DEFAULT_MAX_POSITIONS:
            d["max_position_embeddings"] = self.max_position_embeddings
        if self.eos_token_id >= 0:
            d["eos_token_id"] = self.eos_token_id
        return d

    def save(self, folder: str | Path) -> None:
        write_config_json(folder, self.to_dict())


@register_architecture(ARCHITECTURE, model_types=("vepevik",), config_from_dict=VepevikConfig.from_dict)
def build_vepevik_spec(config: VepevikConfig) -> ModelSpec:
    W, eps = config.width, config.norm_eps

    def norm(name: str) -> PartSpec:
        return PartSpec("rmsnorm", {"dim": W, "eps": eps, "weight": name})

    blending = config.blending_layers
    blocks: list[PartSpec] = []
    ignorable: list[str] = []
    for i, layer in enumerate(config.layers):
        p = f"l{i}."
        if isinstance(layer.mixer, ChunkAttentionConfig):
            leads = len(blending) > 0 and i == blending[0]
            mixer = layer.mixer.part(W, eps, p + "mix.", leads)
            if leads or not layer.mixer.v_mix:
                ignorable.append(p + "mix.vmix")  # a layer that takes in no other layer's values has no use for its share
        else:
            mixer = layer.mixer.part(W, eps, p + "mix.")
        params: dict[str, Any] = {"mixer": mixer, "mixer_norm": norm(p + "norm1")}
        if layer.mlp is not None:
            params.update(feed_forward=layer.mlp.part(W, p + "mlp."), ffn_norm=norm(p + "norm2"))
        else:
            ignorable.append(p + "norm2")  # a layer without a feed-forward has no use for it
        blocks.append(PartSpec("pre_norm", params))
    return ModelSpec(
        vocab_size=config.vocab, hidden_size=W, embedding="embed", layers=blocks, final_norm=norm("final.norm"), lm_head=None,
        max_positions=config.max_position_embeddings, eos_token_id=config.eos_token_id, ignorable_tensors=tuple(ignorable),
        embedding_transform=PartSpec("rmsnorm", {"dim": W, "eps": eps, "weight": "embed.norm"}))


# Named models of this design, so that the command lines can run them with random weights.
for _path in sorted(PRESET_DIR.glob("vepevik-*.json")):
    register_preset("vepevik", _path.stem, _path)
