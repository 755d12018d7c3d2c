"""Typed configuration of the Gezavik decoder, read from its own config.json keys.

config.json of this design is nested: `width`, `vocab`, `norm.eps`, `residual_mult` and a list `layers`, one entry per layer
in running order.  An entry has `type` (which mixer: mamba2 or latent_attention), `mixer` (that mixer's sizes and constants)
and `mlp` (null for none; `kind` dense with `ff`, or `kind` moe with `expert` (`ff`, `limit`), `router` (`experts`, `top`,
`identity`) and `shared` (`ff`, `limit`)).  Every size and constant of a model stands here and nowhere else in the package;
what the design fixes for all of its models stands in the parts' parameters that the model's builder sets.  A key that a
layer may go without (`mask`, `rot`, `vdim`, `groups`, `norm_groups`, `identity`, `shared`, `mlp`) is read as absent.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import List, Optional

from .base import ConfigError, ModelConfig, need_int, opt_float, opt_int
from .padodra import PadodraRotation, _need_dict, _need_float

MIXERS = ("mamba2", "latent_attention")


def _need_positive(raw: dict, key: str, where: str) -> float:
    v = _need_float(raw, key, where)
    if not v > 0:
        raise ConfigError(f"config.json {where}'{key}' = {v} must be positive")
    return v


@dataclass
class GezavikMamba2:
    """`heads` heads of `vdim` channels over states of `state` numbers per channel; B and C in `groups` groups; `conv` taps;
    the gated norm over `norm_groups` equal parts."""
    heads: int
    vdim: int
    state: int
    conv: int
    groups: int = 1
    norm_groups: int = 1

    @classmethod
    def from_dict(cls, raw: dict, where: str) -> "GezavikMamba2":
        heads, vdim = need_int(raw, "heads"), need_int(raw, "vdim")
        groups, norm_groups = opt_int(raw, "groups", 1), opt_int(raw, "norm_groups", 1)
        if heads % groups:
            raise ConfigError(f"config.json {where}'heads' = {heads} is not a multiple of 'groups' = {groups}")
        if (heads * vdim) % norm_groups:
            raise ConfigError(f"config.json {where}'norm_groups' = {norm_groups} does not divide {heads} heads of {vdim}")
        return cls(heads, vdim, need_int(raw, "state"), need_int(raw, "conv"), groups, norm_groups)

    def to_dict(self) -> dict:
        return {"conv": self.conv, "groups": self.groups, "heads": self.heads, "norm_groups": self.norm_groups, "state": self.state,
                "vdim": self.vdim}


@dataclass
class GezavikLatentAttention:
    """`heads` heads of `dim` plain and `rot_dim` rotated query/key dims and `vdim` value dims; queries through a latent of
    `q_rank`, keys and values through one of `kv_rank`; the last `window` tokens are seen (0: all)."""
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    window: int = 0
    rot: Optional[PadodraRotation] = None

    @classmethod
    def from_dict(cls, raw: dict, where: str) -> "GezavikLatentAttention":
        dim, rot_dim = need_int(raw, "dim"), need_int(raw, "rot_dim", minimum=0)
        window = 0
        if raw.get("mask") is not None:
            window = need_int(_need_dict(raw, "mask", where), "size")
        rot = None
        if raw.get("rot") is not None:
            rot = PadodraRotation.from_dict(_need_dict(raw, "rot", where), where + "rot.", rot_dim, ())
        return cls(need_int(raw, "heads"), dim, rot_dim, opt_int(raw, "vdim", dim), need_int(raw, "q_rank"), need_int(raw, "kv_rank"),
                   _need_float(raw, "scale", where), window, rot)

    def to_dict(self) -> dict:
        d = {"dim": self.dim, "heads": self.heads, "kv_rank": self.kv_rank, "q_rank": self.q_rank, "rot_dim": self.rot_dim,
             "scale": self.scale, "vdim": self.vdim}
        if self.window:
            d["mask"] = {"size": self.window}
        if self.rot is not None:
            d["rot"] = self.rot.to_dict()
        return d


_MIXER_CLASSES = {"mamba2": GezavikMamba2, "latent_attention": GezavikLatentAttention}


@dataclass
class GezavikMlp:
    """`kind` dense: `ff`.  `kind` moe: `ff` and `limit` are an expert's, `experts` of them, `identity` further outputs of the
    router, `top` choices per token, and the shared expert's `shared_ff` (0: none) and `shared_limit`."""
    kind: str
    ff: int
    limit: float = 0.0
    experts: int = 0
    top: int = 0
    identity: int = 0
    shared_ff: int = 0
    shared_limit: float = 0.0

    @classmethod
    def from_dict(cls, raw: dict, where: str) -> "GezavikMlp":
        kind = raw.get("kind")
        if kind == "dense":
            return cls("dense", need_int(raw, "ff"))
        if kind != "moe":
            raise ConfigError(f"config.json {where}'kind' = {kind!r} is not supported (supported: dense, moe)")
        r = _need_dict(raw, "router", where)
        experts, top, identity = need_int(r, "experts"), need_int(r, "top"), opt_int(r, "identity", 0, minimum=0)
        if top > experts + identity:
            raise ConfigError(f"config.json {where}router.'top' = {top} exceeds 'experts' = {experts} and 'identity' = {identity}")
        e = _need_dict(raw, "expert", where)
        shared_ff, shared_limit = 0, 0.0
        if raw.get("shared") is not None:
            s = _need_dict(raw, "shared", where)
            shared_ff, shared_limit = need_int(s, "ff"), _need_positive(s, "limit", where + "shared.")
        return cls("moe", need_int(e, "ff"), _need_positive(e, "limit", where + "expert."), experts, top, identity, shared_ff,
                   shared_limit)

    def to_dict(self) -> dict:
        if self.kind == "dense":
            return {"ff": self.ff, "kind": "dense"}
        d = {"expert": {"ff": self.ff, "limit": self.limit}, "kind": "moe",
             "router": {"experts": self.experts, "identity": self.identity, "top": self.top}}
        if self.shared_ff:
            d["shared"] = {"ff": self.shared_ff, "limit": self.shared_limit}
        return d


@dataclass
class GezavikLayer:
    kind: str
    mixer: object
    mlp: Optional[GezavikMlp]


@dataclass
class GezavikConfig(ModelConfig):
    width: int = 0
    vocab: int = 0
    norm_eps: float = 1e-6
    residual_mult: float = 1.0
    layers: List[GezavikLayer] = field(default_factory=list)
    initializer_range: float = 0.05

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    @classmethod
    def from_dict(cls, raw: dict) -> "GezavikConfig":
        width, vocab = need_int(raw, "width"), need_int(raw, "vocab")
        eps = _need_positive(_need_dict(raw, "norm", ""), "eps", "norm.")
        entries = raw.get("layers")
        if not isinstance(entries, list) or not entries:
            raise ConfigError("config.json 'layers' must be a list with at least one layer")
        layers: List[GezavikLayer] = []
        for i, e in enumerate(entries):
            where = f"layers[{i}]."
            if not isinstance(e, dict):
                raise ConfigError(f"config.json layers[{i}] must be an object")
            kind = e.get("type")
            if kind not in MIXERS:
                raise ConfigError(f"config.json {where}'type' = {kind!r} is not supported (supported: {', '.join(MIXERS)})")
            mixer = _MIXER_CLASSES[kind].from_dict(_need_dict(e, "mixer", where), where + "mixer.")
            mlp = None if e.get("mlp") is None else GezavikMlp.from_dict(_need_dict(e, "mlp", where), where + "mlp.")
            layers.append(GezavikLayer(kind, mixer, mlp))
        return cls(architecture="Gezavik", width=width, vocab=vocab, norm_eps=eps, residual_mult=_need_float(raw, "residual_mult", ""),
                   layers=layers, initializer_range=opt_float(raw, "initializer_range", 0.05))

    def to_dict(self) -> dict:
        out = [{"mixer": layer.mixer.to_dict(), "mlp": None if layer.mlp is None else layer.mlp.to_dict(), "type": layer.kind}
               for layer in self.layers]
        return {"architecture": self.architecture, "layers": out, "norm": {"eps": self.norm_eps}, "residual_mult": self.residual_mult,
                "vocab": self.vocab, "width": self.width, "initializer_range": self.initializer_range}
