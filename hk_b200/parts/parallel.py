"""Two mixers side by side: both read the same input, and the layer receives
    left_scale * left(h) + right_scale * right(h).
Either side is any mixer part (an attention over pages beside a recurrent mixer with a state, for instance); the
pair keeps the caches of both, the left one's first.  A side that can carry a factor on its result (it has a
settable `out_scale`: an attention's output gate, a recurrent mixer's output norm) is given its factor when the pair
is made, and then both sides add their output projection straight onto the float32 residual stream.  Otherwise
each side stores its float32 result in a buffer of its own and one kernel adds both, with their factors, onto the
residual stream.  Either way the sum is taken in 32-bit.

With `left_norm` and `right_norm` (RMSNorm parts over the model's width) each result is normed before it takes its factor:
    left_scale * N_l(left(h)) + right_scale * N_r(right(h))
One kernel norms both and adds them onto the residual stream (with the left mixer's output bias, where it has one), and, when
the layer hands it the layer norm of its next sublayer, writes that sublayer's input in the same pass over the row.

Where both sides take their first product from outside (`takes_projection`), their weights over the common input are one
matrix and one product."""
from __future__ import annotations

import torch

from ..csrc import ops
from .base import Part, register_part, stacked_rows
from .norm import LayerNorm


def mixer_cache_specs(mixer) -> list:
    """A mixer's caches as a list: `cache_specs()` where it keeps several, else its one `cache_spec()`."""
    if hasattr(mixer, "cache_specs"):
        return list(mixer.cache_specs())
    return [mixer.cache_spec()]


def mixer_caches(mixer, caches):
    """What a mixer's forward is handed out of `caches` (one per spec): the list, or the single cache."""
    return list(caches) if hasattr(mixer, "cache_specs") else caches[0]


def takes_scale(mixer) -> bool:
    """Whether a mixer or feed-forward carries a factor on its result by itself (set before its tensors are bound)."""
    return hasattr(mixer, "out_scale") and bool(getattr(mixer, "gate", True))      # an attention carries it on its gate


class ParallelMixer(Part):
    graph_safe = True   # reads the batch from device tensors only

    def __init__(self, left, right, left_scale: float = 1.0, right_scale: float = 1.0, left_norm=None, right_norm=None):
        if (left_norm is None) != (right_norm is None):
            raise ValueError("both results are normed, or neither is")
        self.left, self.right, self.left_norm, self.right_norm = left, right, left_norm, right_norm
        self.kernel_libraries = ("norms",) if left_norm is not None else ()
        self._stacked = all(getattr(m, "takes_projection", False) for m in (left, right))
        self.w_in = None
        self.left_scale, self.right_scale = float(left_scale), float(right_scale)
        self._n_left = len(mixer_cache_specs(left))
        self._carried = left_norm is None and all(takes_scale(m) for m in (left, right))
        if self._carried:
            left.out_scale, right.out_scale = self.left_scale, self.right_scale

    @property
    def hidden(self) -> int:
        return self.left.hidden

    def children(self):
        return tuple(p for p in (self.left, self.right, self.left_norm, self.right_norm) if p is not None)

    def bind(self, tensors, precision) -> None:
        super().bind(tensors, precision)
        if self._stacked:           # the sides' own copies become views of the one matrix
            n_left, n_right = int(self.left.in_weight.shape[0]), int(self.right.in_weight.shape[0])
            self.w_in = stacked_rows([stacked_rows([self.left.in_weight], multiple=8), self.right.in_weight], multiple=8)
            at = -(-n_left // 8) * 8            # both sides' columns start aligned for wide loads
            self.left.in_weight, self.right.in_weight = self.w_in[:n_left], self.w_in[at:at + n_right]

    def takes_next_norm(self, norm) -> bool:
        """Whether `forward` can write the layer norm of the new residual stream as well (`next_norm`, `next_out`)."""
        return self.left_norm is not None and isinstance(norm, LayerNorm)

    def cache_specs(self):
        return mixer_cache_specs(self.left) + mixer_cache_specs(self.right)

    def forward(self, xb: torch.Tensor, residual: torch.Tensor, ctx, cache, write_cache: bool = True,
                accumulate: bool = True, next_norm=None, next_out=None) -> None:
        left_cache, right_cache = mixer_caches(self.left, cache[:self._n_left]), mixer_caches(self.right, cache[self._n_left:])
        left_more, right_more = {}, {}
        if self._stacked:
            proj = torch.empty((xb.shape[0], self.w_in.shape[0]), dtype=torch.float32, device=xb.device)
            ops.gemm(xb, self.w_in, proj)
            n_left, n_right = self.left.in_weight.shape[0], self.right.in_weight.shape[0]
            at = -(-n_left // 8) * 8
            left_more["proj"], right_more["proj"] = proj[:, :n_left], proj[:, at:at + n_right]
        if self._carried:
            self.left.forward(xb, residual, ctx, left_cache, write_cache, accumulate=accumulate, **left_more)
            self.right.forward(xb, residual, ctx, right_cache, write_cache, accumulate=True, **right_more)
            return
        y_left = torch.empty(residual.shape, dtype=torch.float32, device=residual.device)
        y_right = torch.empty_like(y_left)
        bias = getattr(self.left, "b_o", None) if self.left_norm is not None else None
        if bias is not None:                    # added by the kernel that norms the result
            left_more["add_bias"] = False
        self.left.forward(xb, y_left, ctx, left_cache, write_cache, accumulate=False, **left_more)
        self.right.forward(xb, y_right, ctx, right_cache, write_cache, accumulate=False, **right_more)
        if self.left_norm is not None:
            ops.pair_norm_add(y_left, self.left_norm.weight, self.left_norm.eps, self.left_scale, y_right, self.right_norm.weight,
                              self.right_norm.eps, self.right_scale, residual, a_bias=bias, accumulate=accumulate,
                              next_norm=(next_norm.weight, next_norm.bias, next_norm.eps) if next_norm is not None else None,
                              next_out=next_out)
            return
        ops.scaled_sum(residual, y_left, self.left_scale, y_right, self.right_scale, accumulate=accumulate)


register_part("mixer", "parallel", ParallelMixer)
