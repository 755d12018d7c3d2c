"""The Nebanex decoder put together from parts, by its configuration.

A layer is pre-norm with layer norms (`PreNormBlock`, `LayerNorm`): x <- x + mixer(N1(x)), x <- x + ff(N2(x)).  The mixer is a
pair side by side (`ParallelMixer`), half the sum of both results, each first RMS-normed over the model's width:

  * left, an attention without a rotation (`GQAAttention`: biases on all four projections, q and k normed over the whole
    projection, a factor on the queries that grows with the position, a learned bias by bucket of distance, an output gate);
  * right, a linear attention with a decay per key channel (`GatedLinearAttention`).

The feed-forward is a mixture of SwiGLU experts (`RoutedFeedForward`: softmax over the chosen logits, a bias on the router)
with a shared expert, or absent.  The embedding is multiplied by `embedding.scale`; the logits come from a matrix of their own
behind the final layer norm and are soft-capped.  Tensor names: `embed`, `l<i>.norm1|norm2` (and `.b`), `l<i>.mix.left.*`,
`l<i>.mix.right.*` (each with `out`, the norm of its result), `l<i>.mlp.*` (`e<j>.`, `shared.`, `router`, `router.b`),
`final.norm`, `head`.
"""
from __future__ import annotations

from ..config import NebanexConfig, register_architecture
from ..parts import (GQAAttention, GatedLinearAttention, LayerNorm, OutputHead, ParallelMixer, PreNormBlock, RMSNorm,
                     RoutedFeedForward, SwiGLUFeedForward, TokenEmbedding)
from ..parts.attention import padded_head
from .spec import ModelSpec

SIDE_SCALE = 0.5            # of each side's normed result
GLU_NAMES = {"gate": "gate", "up": "up", "down": "down"}
ATTENTION_NAMES = {"q": "q", "k": "k", "v": "v", "o": "o", "q_norm": "q.norm", "k_norm": "k.norm", "gate": "g", "rel": "rel",
                   "q_bias": "q.b", "k_bias": "k.b", "v_bias": "v.b", "o_bias": "o.b"}


def _mixer(d: int, layer, prefix: str, eps: float):
    a, r = layer.left, layer.right
    left = GQAAttention(d, a.heads, a.kv_heads, a.dim, prefix + "left.", qk_norm_eps=eps, scale=a.scale, qkv_bias=True, o_bias=True,
                        v_head_dim=a.vdim, gate=True, names=ATTENTION_NAMES, qk_norm_rows=True,
                        q_factor=(a.temp_coef, a.temp_every) if a.temp_every else None, bias_max=a.bias_max,
                        bias_rows=a.bias_rows or None, pad_to=padded_head(a.dim, a.vdim))
    right = GatedLinearAttention(d, r.heads, r.dim, r.vdim, r.tau, prefix + "right.", norm_eps=eps, decay_rank=r.decay_rank or None)
    return ParallelMixer(left, right, SIDE_SCALE, SIDE_SCALE, RMSNorm(d, eps, prefix + "left.out"), RMSNorm(d, eps, prefix + "right.out"))


def _feed_forward(d: int, mlp, prefix: str):
    shared = SwiGLUFeedForward(d, mlp.shared_ff, prefix + "shared.", names=GLU_NAMES) if mlp.shared_ff else None
    return RoutedFeedForward(d, mlp.ff, mlp.experts, mlp.top, prefix, shared=shared, router_bias=True)


def build_nebanex(cfg: NebanexConfig, max_positions: int = 0) -> ModelSpec:
    d, eps = cfg.width, cfg.norm_eps
    blocks = []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        ffn = ffn_norm = None
        if layer.mlp is not None:
            ffn, ffn_norm = _feed_forward(d, layer.mlp, p + "mlp."), LayerNorm(d, eps, p + "norm2")
        blocks.append(PreNormBlock(LayerNorm(d, eps, p + "norm1"), _mixer(d, layer, p + "mix.", eps), ffn_norm, ffn))
    embedding = TokenEmbedding(cfg.vocab, d, "embed", scale=cfg.embedding_scale)
    head = OutputHead(d, cfg.vocab, LayerNorm(d, eps, "final.norm"), "head", softcap=cfg.logit_softcap)
    return ModelSpec(cfg, embedding, blocks, head)


register_architecture("Nebanex", NebanexConfig, build_nebanex, "nebanex")
