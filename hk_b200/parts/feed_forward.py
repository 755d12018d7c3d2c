"""SwiGLU feed-forward: residual += (silu(xb Wg^T) * (xb Wu^T)) Wd^T, no biases
(src/engine/cpu_backend.zig:308-323, src/engine/ops.zig:65-80).  Gate and up are one
product over the concatenated weight [2F, d] (the reference fuses them into one parallel
region: src/engine/matmul.zig:93-96).  The gate's activation is a parameter (`act`: silu, or gelu_tanh =
0.5 z (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3))), which makes it a GeGLU), and so are the tensors' names.
`act="swish_clamped"` is the clamped form: with g = min(gate, limit) and u = clamp(up, -limit, limit) the hidden
vector is g * sigmoid(slope * g) * (u + 1); `limit` and `slope` are parameters."""
from __future__ import annotations

from typing import Dict

import torch

from ..csrc import ops
from .base import MATRIX, VECTOR, ParamSpec, Part, Precision, register_part


class SwiGLUFeedForward(Part):
    graph_safe = True   # reads the batch from device tensors only

    def __init__(self, hidden: int, intermediate: int, prefix: str, act: str = "silu", names=None, limit: float = 0.0,
                 slope: float = 1.0):
        if act not in ops.GLU_ACTS:
            raise ValueError(f"activation '{act}' is not one of {', '.join(ops.GLU_ACTS)}")
        if act == "swish_clamped" and not limit > 0:
            raise ValueError("the clamped activation needs a positive limit")
        self.hidden, self.F, self.prefix, self.act = hidden, intermediate, prefix, act
        self.limit, self.slope = float(limit), float(slope)
        self.names = {"gate": "gate_proj.weight", "up": "up_proj.weight", "down": "down_proj.weight"}
        self.names.update(names or {})
        self.w_gate_up = self.w_down = None

    def own_param_specs(self) -> Dict[str, ParamSpec]:
        p, nm = self.prefix, self.names
        return {
            p + nm["gate"]: ParamSpec((self.F, self.hidden), MATRIX),
            p + nm["up"]: ParamSpec((self.F, self.hidden), MATRIX),
            p + nm["down"]: ParamSpec((self.hidden, self.F), MATRIX),
        }

    def own_bind(self, tensors, precision: Precision) -> None:
        p, nm = self.prefix, self.names
        gate, up = tensors[p + nm["gate"]], tensors[p + nm["up"]]
        # One matrix [all gate rows | all up rows]: one product gives both halves, and the tensor-core kernels take a
        # tile's rows half from each so that SwiGLU runs in their epilogue (cf. the reference's fused gate/up product,
        # shaders/swiglu_pair.comp:2).
        if gate.dtype != up.dtype:                  # one of them kept in 32-bit: both are
            gate, up = gate.float(), up.float()
        self.w_gate_up = torch.cat([gate, up], dim=0).contiguous()
        self.w_down = tensors[p + nm["down"]]

    def forward(self, xb: torch.Tensor, residual: torch.Tensor, ctx, accumulate: bool = True) -> None:
        h = torch.empty((xb.shape[0], self.F), dtype=xb.dtype, device=xb.device)
        ops.gemm_swiglu(xb, self.w_gate_up, h, self.act, self.limit, self.slope)
        ops.gemm(h, self.w_down, residual, accumulate=accumulate)


register_part("feed_forward", "swiglu", SwiGLUFeedForward)


class SquaredReLUFeedForward(Part):
    """residual += out_scale * W_down max(W_up xb, 0)^2, no gate and no biases; the activation (with the factor) runs in the
    epilogue of the up product where a tensor-core product takes it."""
    graph_safe = True   # reads the batch from device tensors only

    def __init__(self, hidden: int, intermediate: int, prefix: str, names=None, out_scale: float = 1.0):
        self.hidden, self.F, self.prefix, self.out_scale = hidden, intermediate, prefix, float(out_scale)
        self.names = {"up": "up", "down": "down"}
        self.names.update(names or {})
        self.w_up = self.w_down = None

    def own_param_specs(self) -> Dict[str, ParamSpec]:
        p, nm = self.prefix, self.names
        return {p + nm["up"]: ParamSpec((self.F, self.hidden), MATRIX), p + nm["down"]: ParamSpec((self.hidden, self.F), MATRIX)}

    def own_bind(self, tensors, precision: Precision) -> None:
        self.w_up, self.w_down = tensors[self.prefix + self.names["up"]], tensors[self.prefix + self.names["down"]]

    def forward(self, xb: torch.Tensor, residual: torch.Tensor, ctx, accumulate: bool = True) -> None:
        h = torch.empty((xb.shape[0], self.F), dtype=xb.dtype, device=xb.device)
        ops.gemm_squared_relu(xb, self.w_up, h, self.out_scale)
        ops.gemm(h, self.w_down, residual, accumulate=accumulate)


class PolyNormFeedForward(Part):
    """residual += W_down act(W_up xb) with the polynomial activation
        act(z) = c0 N(z) + c1 N(z^2) + c2 N(z^3) + c3,   N(v) = v / sqrt(mean(v^2) + eps) over a token's F values,
    powers element by element; the four numbers are a tensor of the model (`act`).  The up product's result is
    float32, the three means and the activation are computed in float32 and narrowed for the down product."""
    graph_safe = True   # reads the batch from device tensors only

    def __init__(self, hidden: int, intermediate: int, prefix: str, eps: float, names=None):
        self.hidden, self.F, self.prefix, self.eps = hidden, intermediate, prefix, float(eps)
        self.names = {"up": "up", "down": "down", "act": "act"}
        self.names.update(names or {})
        self.w_up = self.w_down = self.coef = None

    def own_param_specs(self) -> Dict[str, ParamSpec]:
        p, nm = self.prefix, self.names
        return {
            p + nm["up"]: ParamSpec((self.F, self.hidden), MATRIX),
            p + nm["down"]: ParamSpec((self.hidden, self.F), MATRIX),
            p + nm["act"]: ParamSpec((4,), VECTOR, "one_plus_normal"),
        }

    def own_bind(self, tensors, precision: Precision) -> None:
        p, nm = self.prefix, self.names
        self.w_up, self.w_down, self.coef = tensors[p + nm["up"]], tensors[p + nm["down"]], tensors[p + nm["act"]]

    def forward(self, xb: torch.Tensor, residual: torch.Tensor, ctx, accumulate: bool = True) -> None:
        n = xb.shape[0]
        z = torch.empty((n, self.F), dtype=torch.float32, device=xb.device)
        ops.gemm(xb, self.w_up, z)
        h = torch.empty((n, self.F), dtype=xb.dtype, device=xb.device)
        ops.polynorm(z, self.coef, self.eps, h)
        ops.gemm(h, self.w_down, residual, accumulate=accumulate)


class RoutedFeedForward(Part):
    """A mixture of `experts` SwiGLU feed-forwards of which every token uses `top`:
        router logits z = W_router xb in float32; the `top` largest are chosen (the lower index wins a tie) and
        weighted by the softmax over the chosen logits; residual += sum_k weight_k * W_down_e (silu(W_gate_e xb) * W_up_e xb).
    The choice never leaves the device (`csrc/routed.cu`): tokens are sorted by expert there and the experts'
    products run as one grouped product over tiles of the sorted rows, so the launches depend on the number of
    rows alone.  The experts' weights are stacked at binding: [E, 2F, d] (gate rows, then up rows) and [E, d, F].

    `scores="sigmoid"` is another router: every expert's score is s = sigmoid(z) by itself; the choice is made on
    s + correction (`correction=True`: a tensor [E] of the model, used for the choice alone), among the experts of the best
    `keep` of `groups` equal groups of neighbours when `groups` is given (a group's score is the sum of its two largest
    choice scores; the experts of the other groups count as minus infinity), and the weights are the chosen experts' s over
    their sum + `norm_eps`, times `weight_scale`.  `shared`: one more feed-forward part that every token uses; its result is
    added to the experts' sum, times sigmoid(W_sg xb) (one number per token, tensor `shared_gate` [1, d], whose product
    rides along with the router's in 32-bit) when `shared_gated` is set.

    `scores="softmax_all"` is a third router: s = softmax(z) over all of its outputs, the choice is made on s + correction,
    and the weights are the chosen s themselves (times `weight_scale`).  `identity`: the router has that many further
    outputs behind the experts' which stand for no feed-forward: such a choice gives back xb itself, times its weight.
    `router_bias`: a tensor with one entry per router output that is added to the logits (for every kind of scores).
    `act`, `limit`, `slope` are the experts' gated activation (silu, or the clamped form of `SwiGLUFeedForward`);
    `out_scale` is a factor on the whole result."""
    graph_safe = True   # reads the batch from device tensors only; launches depend on the row count alone
    kernel_libraries = ("routed",)
    route_log = None    # a list, when someone wants to see the choices: every eager forward appends a copy of its
                        # chosen experts int32 [rows, top] (a replayed graph runs no Python and appends nothing)

    def __init__(self, hidden: int, intermediate: int, n_experts: int, top: int, prefix: str, names=None,
                 scores: str = "softmax", correction: bool = False, groups: int = 0, keep: int = 0, weight_scale: float = 1.0,
                 norm_eps: float = 0.0, shared=None, shared_gated: bool = False, identity: int = 0, act: str = "silu",
                 limit: float = 0.0, slope: float = 1.0, out_scale: float = 1.0, router_bias: bool = False):
        if identity < 0 or not 1 <= top <= n_experts + identity or top > 32:
            raise ValueError(f"top = {top} must be in 1..min(experts, 32) (experts = {n_experts}, identities = {identity})")
        if scores not in ops.ROUTE_SCORES:
            raise ValueError(f"scores '{scores}' is not one of {', '.join(ops.ROUTE_SCORES)}")
        if scores == "softmax_all" and (groups or shared_gated):
            raise ValueError("groups and a gated shared part belong to scores='sigmoid'")
        if act not in ("silu", "swish_clamped") or (act == "swish_clamped" and not limit > 0):
            raise ValueError("the experts' activation is 'silu', or 'swish_clamped' with a positive limit")
        if scores == "softmax" and (correction or groups or weight_scale != 1.0 or shared_gated):
            raise ValueError("a correction, groups, a factor on the weights and a gated shared part belong to scores='sigmoid'")
        if groups and (n_experts % groups or not 1 <= keep <= groups):
            raise ValueError(f"{n_experts} experts do not form {groups} equal groups of which {keep} are kept")
        if router_bias and shared_gated:
            raise ValueError("the gate of a shared part is a row of the router's product and has no bias")
        if shared_gated and shared is None:
            raise ValueError("shared_gated needs a shared part")
        self.hidden, self.F, self.E, self.top, self.prefix = hidden, intermediate, n_experts, top, prefix
        self.scores, self.correction, self.groups, self.keep = scores, bool(correction), int(groups), int(keep)
        self.weight_scale, self.norm_eps = float(weight_scale), float(norm_eps)
        self.shared, self.shared_gated = shared, bool(shared_gated)
        self.identity, self.act, self.limit, self.slope = int(identity), act, float(limit), float(slope)
        self.out_scale, self.router_bias = float(out_scale), bool(router_bias)
        self.names = {"router": "router", "router_bias": "router.b", "expert": "e{}.", "gate": "gate", "up": "up", "down": "down",
                      "correction": "correction", "shared_gate": "shared.sg"}
        self.names.update(names or {})
        self.w_router = self.w_gate_up = self.w_down = self.w_correction = self.b_router = None

    def children(self):
        return (self.shared,) if self.shared is not None else ()

    def _expert(self, e: int, which: str) -> str:
        return self.prefix + self.names["expert"].format(e) + self.names[which]

    def own_param_specs(self) -> Dict[str, ParamSpec]:
        outputs = self.E + self.identity
        specs = {self.prefix + self.names["router"]: ParamSpec((outputs, self.hidden), MATRIX)}
        if self.router_bias:
            specs[self.prefix + self.names["router_bias"]] = ParamSpec((outputs,), VECTOR)
        if self.correction:
            specs[self.prefix + self.names["correction"]] = ParamSpec((outputs,), VECTOR)
        if self.shared_gated:
            specs[self.prefix + self.names["shared_gate"]] = ParamSpec((1, self.hidden), MATRIX)
        for e in range(self.E):
            specs[self._expert(e, "gate")] = ParamSpec((self.F, self.hidden), MATRIX)
            specs[self._expert(e, "up")] = ParamSpec((self.F, self.hidden), MATRIX)
            specs[self._expert(e, "down")] = ParamSpec((self.hidden, self.F), MATRIX)
        return specs

    def own_bind(self, tensors, precision: Precision) -> None:
        self.w_router = tensors[self.prefix + self.names["router"]].float().contiguous()    # the router runs in 32-bit
        if self.shared_gated:       # the shared part's gate is one more row of the router's product
            self.w_router = torch.cat([self.w_router, tensors[self.prefix + self.names["shared_gate"]].float()]).contiguous()
        if self.router_bias:
            self.b_router = tensors[self.prefix + self.names["router_bias"]]
        if self.correction:
            self.w_correction = tensors[self.prefix + self.names["correction"]]
        dt = precision.compute
        self.w_gate_up = torch.stack([torch.cat([tensors[self._expert(e, "gate")].to(dt), tensors[self._expert(e, "up")].to(dt)])
                                      for e in range(self.E)]).contiguous()
        self.w_down = torch.stack([tensors[self._expert(e, "down")].to(dt) for e in range(self.E)]).contiguous()
        self._tile_rows = ops.route_tile_rows()

    TC_MIN_PAIRS = 1024     # from this many (row, choice) pairs on, a bfloat16 step takes the tcgen05 grouped product

    def _forward_tc(self, xb, residual, ids, weights, accumulate: bool, shared_y=None, shared_gate=None) -> bool:
        """Prompt-sized steps in bfloat16: the rows are gathered into expert order with every expert's rows padded to whole
        128-row tiles, and both products run on the tcgen05 kernel with a tile's expert choosing its weights."""
        from ..csrc import gemm_fast
        n, dev = xb.shape[0], xb.device
        pairs, pad = n * self.top, gemm_fast.GROUPED_ROWS
        m_max = -(-(pairs + self.E * (pad - 1)) // pad) * pad
        perm = torch.empty(m_max, dtype=torch.int32, device=dev)
        inv = torch.empty(pairs, dtype=torch.int32, device=dev)
        groups = torch.empty(m_max // pad, dtype=torch.int32, device=dev)
        ops.route_sort_padded(ids, self.E, pad, perm, inv, groups)
        xs = torch.empty((m_max, self.hidden), dtype=xb.dtype, device=dev)
        ops.route_gather(xb, perm, self.top, xs)
        h = torch.empty((m_max, self.F), dtype=xb.dtype, device=dev)
        if not ops.grouped_gemm_tc(xs, self.w_gate_up, h, groups, gated=True, act=self.act, limit=self.limit, slope=self.slope):
            return False
        ys = torch.empty((m_max, self.hidden), dtype=torch.float32, device=dev)
        if not ops.grouped_gemm_tc(h, self.w_down, ys, groups, gated=False):
            return False
        self._combine(ys, inv, weights, xb, residual, accumulate, shared_y, shared_gate)
        return True

    def _combine(self, ys, inv, weights, xb, residual, accumulate: bool, shared_y, shared_gate) -> None:
        ops.route_combine(ys, inv, weights, residual, accumulate=accumulate, shared=shared_y, shared_gate=shared_gate,
                          x=xb if self.identity else None, factor=self.out_scale)

    def forward(self, xb: torch.Tensor, residual: torch.Tensor, ctx, accumulate: bool = True) -> None:
        n, dev = xb.shape[0], xb.device
        pairs = n * self.top
        ids = torch.empty((n, self.top), dtype=torch.int32, device=dev)
        weights = torch.empty((n, self.top), dtype=torch.float32, device=dev)
        shared_gate = torch.empty((n, 1), dtype=torch.float32, device=dev) if self.shared_gated else None
        ops.route_topk(xb, self.w_router, ids, weights, self.scores, self.w_correction, self.groups, self.keep, self.weight_scale,
                       self.norm_eps, shared_gate, self.b_router)
        if RoutedFeedForward.route_log is not None:
            RoutedFeedForward.route_log.append(ids.clone())
        shared_y = None
        if self.shared is not None:
            shared_y = torch.empty((n, self.hidden), dtype=torch.float32, device=dev)
            self.shared.forward(xb, shared_y, ctx, accumulate=False)
        if xb.dtype == torch.bfloat16 and pairs >= self.TC_MIN_PAIRS and self.hidden % 8 == 0 and self.F % 8 == 0 \
                and self._forward_tc(xb, residual, ids, weights, accumulate, shared_y, shared_gate):
            return
        max_tiles = pairs // self._tile_rows + min(self.E, pairs)
        offsets = torch.empty(self.E + 1, dtype=torch.int32, device=dev)
        perm = torch.empty(pairs, dtype=torch.int32, device=dev)
        inv = torch.empty(pairs, dtype=torch.int32, device=dev)
        tiles = torch.empty((max_tiles, 2), dtype=torch.int32, device=dev)
        ops.route_sort(ids, self.E, offsets, perm, inv, tiles)
        h = torch.empty((pairs, self.F), dtype=xb.dtype, device=dev)
        ops.grouped_gemm(xb, self.w_gate_up, h, tiles, offsets, perm, self.top, gather=True, gated=True, act=self.act,
                         limit=self.limit, slope=self.slope)
        ys = torch.empty((pairs, self.hidden), dtype=torch.float32, device=dev)
        ops.grouped_gemm(h, self.w_down, ys, tiles, offsets, perm, self.top, gather=False, gated=False)
        self._combine(ys, inv, weights, xb, residual, accumulate, shared_y, shared_gate)


register_part("feed_forward", "squared_relu", SquaredReLUFeedForward)
register_part("feed_forward", "polynorm", PolyNormFeedForward)
register_part("feed_forward", "routed_swiglu", RoutedFeedForward)
