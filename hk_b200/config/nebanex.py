"""Typed configuration of the Nebanex decoder, read from its own config.json keys.

config.json of this design is nested: `width`, `vocab`, `norm.eps`, `embedding.scale`, `logit_softcap` and a list `layers`,
one entry per layer in running order.  An entry has `type` (parallel), `mixer` (the sizes and constants of its two sides
under `left` and `right`) and `mlp` (null for none; `kind` moe with `expert.ff`, `router.experts`, `router.top` and
`shared.ff`).  The left side is an attention: `heads`, `kv_heads`, `dim`, `vdim`, `scale`, `bias_max` (how far its distance
bias is resolved) and `q_temp` (`coef`, `every`; absent: the queries take no factor); the right side a gated linear
attention: `heads`, `dim`, `vdim`, `tau`.  The rows of the distance bias and the width of the decay's low-rank projection
are in no key: a file's tensors give them (`bias_rows` and `decay_rank` may stand in the configuration for a model whose
weights are made at random).  Every size and constant of a model stands here and nowhere else in the package; what the
design fixes for all of its models stands in the parts and in the model's builder.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import List, Optional

from .base import ConfigError, ModelConfig, need_int, opt_float, opt_int
from .padodra import _need_dict, _need_float, _opt_positive

MIXERS = ("parallel",)


def _need_positive(raw: dict, key: str, where: str) -> float:
    v = _need_float(raw, key, where)
    if not v > 0:
        raise ConfigError(f"config.json {where}'{key}' = {v} must be positive")
    return v


def _as_given(v: float):
    return int(v) if float(v).is_integer() else v


@dataclass
class NebanexAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    bias_max: float
    temp_coef: float = 0.0
    temp_every: int = 0             # 0: no factor on the queries
    bias_rows: int = 0              # 0: as the file's tensor has it

    @classmethod
    def from_dict(cls, raw: dict, where: str) -> "NebanexAttention":
        heads, dim = need_int(raw, "heads"), need_int(raw, "dim")
        kv_heads = opt_int(raw, "kv_heads", heads)
        if heads % kv_heads:
            raise ConfigError(f"config.json {where}'heads' = {heads} is not a multiple of 'kv_heads' = {kv_heads}")
        coef, every = 0.0, 0
        if raw.get("q_temp") is not None:
            t = _need_dict(raw, "q_temp", where)
            coef, every = _need_float(t, "coef", where + "q_temp."), need_int(t, "every")
        return cls(heads, kv_heads, dim, opt_int(raw, "vdim", dim), _need_float(raw, "scale", where),
                   _need_positive(raw, "bias_max", where), coef, every, opt_int(raw, "bias_rows", 0))

    def to_dict(self) -> dict:
        d = {"bias_max": _as_given(self.bias_max), "dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "scale": self.scale,
             "vdim": self.vdim}
        if self.temp_every:
            d["q_temp"] = {"coef": self.temp_coef, "every": self.temp_every}
        if self.bias_rows:
            d["bias_rows"] = self.bias_rows
        return d


@dataclass
class NebanexLinear:
    heads: int
    dim: int
    vdim: int
    tau: float
    decay_rank: int = 0             # 0: as the file's tensor has it

    @classmethod
    def from_dict(cls, raw: dict, where: str) -> "NebanexLinear":
        dim = need_int(raw, "dim")
        return cls(need_int(raw, "heads"), dim, opt_int(raw, "vdim", dim), _need_positive(raw, "tau", where), opt_int(raw, "decay_rank", 0))

    def to_dict(self) -> dict:
        d = {"dim": self.dim, "heads": self.heads, "tau": self.tau, "vdim": self.vdim}
        if self.decay_rank:
            d["decay_rank"] = self.decay_rank
        return d


@dataclass
class NebanexMlp:
    """`experts` feed-forwards of size `ff`, `top` choices per token, and the shared expert's `shared_ff` (0: none)."""
    ff: int
    experts: int
    top: int
    shared_ff: int = 0

    @classmethod
    def from_dict(cls, raw: dict, where: str) -> "NebanexMlp":
        if raw.get("kind") != "moe":
            raise ConfigError(f"config.json {where}'kind' = {raw.get('kind')!r} is not supported (supported: moe)")
        r = _need_dict(raw, "router", where)
        experts, top = need_int(r, "experts"), need_int(r, "top")
        if top > experts:
            raise ConfigError(f"config.json {where}router.'top' = {top} exceeds 'experts' = {experts}")
        shared_ff = need_int(_need_dict(raw, "shared", where), "ff") if raw.get("shared") is not None else 0
        return cls(need_int(_need_dict(raw, "expert", where), "ff"), experts, top, shared_ff)

    def to_dict(self) -> dict:
        d = {"expert": {"ff": self.ff}, "kind": "moe", "router": {"experts": self.experts, "top": self.top}}
        if self.shared_ff:
            d["shared"] = {"ff": self.shared_ff}
        return d


@dataclass
class NebanexLayer:
    left: NebanexAttention
    right: NebanexLinear
    mlp: Optional[NebanexMlp]


@dataclass
class NebanexConfig(ModelConfig):
    width: int = 0
    vocab: int = 0
    norm_eps: float = 1e-6
    embedding_scale: float = 1.0
    logit_softcap: float = 0.0                  # 0: none
    layers: List[NebanexLayer] = field(default_factory=list)
    initializer_range: float = 0.05

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    @classmethod
    def from_dict(cls, raw: dict) -> "NebanexConfig":
        width, vocab = need_int(raw, "width"), need_int(raw, "vocab")
        eps = _need_positive(_need_dict(raw, "norm", ""), "eps", "norm.")
        emb_scale = 1.0
        if raw.get("embedding") is not None:
            emb_scale = opt_float(_need_dict(raw, "embedding", ""), "scale", 1.0)
        entries = raw.get("layers")
        if not isinstance(entries, list) or not entries:
            raise ConfigError("config.json 'layers' must be a list with at least one layer")
        layers: List[NebanexLayer] = []
        for i, e in enumerate(entries):
            where = f"layers[{i}]."
            if not isinstance(e, dict):
                raise ConfigError(f"config.json layers[{i}] must be an object")
            if e.get("type") not in MIXERS:
                raise ConfigError(f"config.json {where}'type' = {e.get('type')!r} is not supported (supported: {', '.join(MIXERS)})")
            m = _need_dict(e, "mixer", where)
            left = NebanexAttention.from_dict(_need_dict(m, "left", where + "mixer."), where + "mixer.left.")
            right = NebanexLinear.from_dict(_need_dict(m, "right", where + "mixer."), where + "mixer.right.")
            mlp = None if e.get("mlp") is None else NebanexMlp.from_dict(_need_dict(e, "mlp", where), where + "mlp.")
            layers.append(NebanexLayer(left, right, mlp))
        return cls(architecture="Nebanex", width=width, vocab=vocab, norm_eps=eps, embedding_scale=emb_scale,
                   logit_softcap=_opt_positive(raw, "logit_softcap", ""), layers=layers,
                   initializer_range=opt_float(raw, "initializer_range", 0.05))

    def to_dict(self) -> dict:
        out = [{"mixer": {"left": layer.left.to_dict(), "right": layer.right.to_dict()},
                "mlp": None if layer.mlp is None else layer.mlp.to_dict(), "type": "parallel"} for layer in self.layers]
        d = {"architecture": self.architecture, "embedding": {"scale": self.embedding_scale}, "layers": out,
             "norm": {"eps": self.norm_eps}, "vocab": self.vocab, "width": self.width, "initializer_range": self.initializer_range}
        if self.logit_softcap:
            d["logit_softcap"] = self.logit_softcap
        return d
