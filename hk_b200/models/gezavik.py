"""The Gezavik decoder put together from parts, by its configuration.

A layer has one norm, and its two sublayers stand side by side on the norm's output (`ParallelBlock`):
x <- x + residual_mult * (mixer(N(x)) + ff(N(x))).  The mixer is, layer by layer,

  * `mamba2`: a state-space recurrence behind a short convolution (`StateSpace`), its output gated before a norm over equal
    parts;
  * `latent_attention`: attention over one cached vector per token (`LatentAttention`) with queries through a latent of their
    own, a rotated part in adjacent pairs, a sliding window and one sigmoid gate per head.

The feed-forward is dense with a squared relu (`SquaredReLUFeedForward`), a mixture of experts with the clamped activation
(`RoutedFeedForward`: softmax over all of the router's outputs, a correction for the choice alone, weights as they are,
identity outputs, and a shared expert with a limit of its own), or absent.  The logits come from a matrix of their own behind
the final norm.  Tensor names: `embed`, `l<i>.norm1`, `l<i>.mix.*`, `l<i>.mlp.*` (`e<j>.`, `shared.`, `router`,
`correction`), `final.norm`, `head`.
"""
from __future__ import annotations

from ..config import GezavikConfig, register_architecture
from ..parts import (LatentAttention, OutputHead, ParallelBlock, RMSNorm, RotaryEmbedding, RoutedFeedForward,
                     SquaredReLUFeedForward, StateSpace, SwiGLUFeedForward, TokenEmbedding)
from .spec import ModelSpec

SWISH_SLOPE = 1.702         # the sigmoid's slope in the experts' activation
GLU_NAMES = {"gate": "gate", "up": "up", "down": "down"}


def _rotation(rot, positions: int, made: dict):
    if rot is None:
        return None
    key = (rot.base, rot.dims)
    if key not in made:
        made[key] = RotaryEmbedding(rot.base, rot.dims, positions, pairing="adjacent")
    return made[key]


def _feed_forward(d: int, mlp, prefix: str):
    if mlp.kind == "dense":
        return SquaredReLUFeedForward(d, mlp.ff, prefix)
    shared = None
    if mlp.shared_ff:
        shared = SwiGLUFeedForward(d, mlp.shared_ff, prefix + "shared.", act="swish_clamped", names=GLU_NAMES, limit=mlp.shared_limit,
                                   slope=SWISH_SLOPE)
    return RoutedFeedForward(d, mlp.ff, mlp.experts, mlp.top, prefix, scores="softmax_all", correction=True, identity=mlp.identity,
                             act="swish_clamped", limit=mlp.limit, slope=SWISH_SLOPE, shared=shared)


def build_gezavik(cfg: GezavikConfig, max_positions: int = 0) -> ModelSpec:
    d, eps = cfg.width, cfg.norm_eps
    positions = max(int(max_positions), 1)
    ropes: dict = {}
    blocks = []
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer.mixer
        if layer.kind == "mamba2":
            mixer = StateSpace(d, m.heads, m.vdim, m.state, m.groups, m.conv, p + "mix.", eps, norm_groups=m.norm_groups)
        else:
            mixer = LatentAttention(d, m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank, p + "mix.", eps, m.scale,
                                    position=_rotation(m.rot, positions, ropes), gate="head", window=m.window or None, q_rank=m.q_rank)
        ffn = None if layer.mlp is None else _feed_forward(d, layer.mlp, p + "mlp.")
        blocks.append(ParallelBlock(RMSNorm(d, eps, p + "norm1"), mixer, ffn, cfg.residual_mult))
    embedding = TokenEmbedding(cfg.vocab, d, "embed")
    head = OutputHead(d, cfg.vocab, RMSNorm(d, eps, "final.norm"), "head")
    return ModelSpec(cfg, embedding, blocks, head)


register_architecture("Gezavik", GezavikConfig, build_gezavik, "gezavik")
