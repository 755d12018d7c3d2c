"""Tiny Nebanex configurations for the tests: layers in several shapes, with and without the keys a layer may go without (query
factor, shared expert, feed-forward, soft cap), and sizes chosen so that nothing that could be confused is equal (heads and
key/value heads, key and value sizes, the two mixers' sizes, bias rows and reach, experts and choices) or happens to be 1 by
accident.  The distance biases, the routers' rows and biases and the decays' biases are made larger than the other weights, so
that none of them is flat; the soft caps are near the logits' size."""
from __future__ import annotations

import json
import os

import numpy as np
import torch

import helpers


def left(heads, kv_heads, dim, vdim, scale, bias_max, bias_rows, q_temp=None):
    m = {"bias_max": bias_max, "bias_rows": bias_rows, "dim": dim, "heads": heads, "kv_heads": kv_heads, "scale": scale, "vdim": vdim}
    if q_temp:
        m["q_temp"] = {"coef": q_temp[0], "every": q_temp[1]}
    return m


def right(heads, dim, vdim, tau, rank):
    return {"decay_rank": rank, "dim": dim, "heads": heads, "tau": tau, "vdim": vdim}


def moe(ff, experts, top, shared=0):
    m = {"expert": {"ff": ff}, "kind": "moe", "router": {"experts": experts, "top": top}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def layer(lhs, rhs, mlp):
    return {"type": "parallel", "mixer": {"left": lhs, "right": rhs}, "mlp": mlp}


def config(width, vocab, eps, scale, cap, layers, std):
    c = {"architecture": "Nebanex", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": scale}, "layers": layers,
         "initializer_range": std}
    if cap:
        c["logit_softcap"] = cap
    return c


CONFIGS = {
    # heads of sizes no tensor-core kernel knows (filled up to 64), keys and values of different size; a feed-forward with all
    # experts but one chosen; a layer without a feed-forward
    "A": config(48, 131, 1e-6, 1.5, 2.5, [
        layer(left(6, 2, 10, 6, 0.3, 20, 6, (0.7, 9)), right(3, 8, 12, 4.0, 5), moe(24, 5, 2, 40)),
        layer(left(4, 4, 12, 20, 0.25, 50, 10), right(2, 16, 4, 1.0, 8), None),
        layer(left(3, 1, 6, 9, 0.4, 9, 4, (-0.2, 3)), right(5, 12, 8, 16.0, 3), moe(16, 4, 3)),
    ], 0.12),
    # head sizes of the mma.sync kernels as they are; value columns and states that no vector load divides
    "B": config(64, 200, 1e-5, 0.8, 4.0, [
        layer(left(4, 2, 16, 16, 0.3, 40, 8, (0.4, 16)), right(3, 10, 5, 8.0, 4), moe(24, 6, 4, 32)),
        layer(left(6, 6, 32, 32, 0.2, 17, 12, (0.5, 25)), right(2, 34, 21, 3.0, 16), moe(32, 3, 1)),
    ], 0.1),
    # the tensor-core kernels' sizes: heads of 64 and of 128 (values of 40 filled up), states of 64 and 128, expert sizes of the
    # grouped tcgen05 product
    "C": config(128, 300, 1e-5, 1.2, 3.0, [
        layer(left(8, 2, 64, 64, 0.12, 100, 16, (0.5, 40)), right(2, 64, 48, 16.0, 16), moe(40, 6, 3, 64)),
        layer(left(6, 3, 128, 40, 0.1, 70, 32, (0.3, 64)), right(1, 128, 72, 5.0, 12), moe(48, 8, 2, 24)),
    ], 0.08),
    # a head above 128 (the generic attention kernel in either type), one head, one row of bias beside two, no soft cap; widths
    # that are no multiple of 4 or 8; a factor that changes at every position
    "D": config(42, 103, 1e-6, 1.0, 0.0, [
        layer(left(2, 1, 130, 7, 0.08, 12, 5, (0.15, 1)), right(1, 21, 34, 2.0, 1), moe(12, 2, 2, 20)),
        layer(left(1, 1, 5, 13, 0.4, 3, 2), right(3, 7, 3, 1.0, 9), moe(20, 6, 1)),
        layer(left(3, 3, 4, 4, 0.5, 7, 1, (1.1, 50)), right(2, 200, 6, 11.0, 6), None),
    ], 0.15),
}
SEEDS = {"A": 71, "B": 77, "C": 73, "D": 74}
# tensors whose names end so: value * factor + shift
SHARPEN = {".rel": (14.0, 0.0), ".router": (3.0, 0.0), ".router.b": (6.0, 0.0), ".a2.b": (12.0, 1.5), ".a1": (2.0, 0.0), ".a2": (3.0, 0.0),
           "norm1.b": (2.0, 0.0), "norm2.b": (2.0, 0.0), "final.norm.b": (3.0, 0.0), ".o.b": (3.0, 0.0)}


def make_model_dir(tmpdir, which: str, dtype=torch.float32) -> str:
    """Seeded random weights of configuration `which`, some of them sharpened; matrices stored as `dtype`."""
    from hk_b200.config import config_from_dict, resolve_architecture
    from hk_b200.weights import random_tensors
    from hk_b200.weights.safetensors_io import save_file
    raw = CONFIGS[which]
    cfg = config_from_dict(raw)
    _, build = resolve_architecture(cfg.architecture)
    specs = build(cfg, 8).param_specs()
    tensors = random_tensors(specs, SEEDS[which], raw["initializer_range"], 0.1, "cuda" if torch.cuda.is_available() else "cpu",
                             dtype_of=lambda s: torch.float32 if s.kind == "vector" else dtype)
    tensors = {k: v.cpu() for k, v in tensors.items()}
    for name in tensors:
        for ending, (factor, shift) in SHARPEN.items():
            if name.endswith(ending):
                tensors[name] = (tensors[name].float() * factor + shift).to(tensors[name].dtype)
    d = os.path.join(str(tmpdir), f"nebanex_{which}_{str(dtype).split('.')[-1]}")
    os.makedirs(d, exist_ok=True)
    with open(os.path.join(d, "config.json"), "w", encoding="utf-8") as f:
        json.dump(cfg.to_dict(), f, indent=1)
    save_file(tensors, os.path.join(d, "model.safetensors"))
    return d


def prompts(which: str, rng: np.random.Generator, lengths):
    return [rng.integers(0, CONFIGS[which]["vocab"], n).tolist() for n in lengths]


def routed_prefixes(cfg: dict):
    """The tensor prefixes of the routed feed-forwards, in running order."""
    return [f"l{i}.mlp." for i, e in enumerate(cfg["layers"]) if e.get("mlp")]


def load_plain(d):
    """The folder's configuration and float64 weights; a model without a soft cap has one that no logit feels."""
    cfg, w = helpers.load_plain(d)
    cfg.setdefault("logit_softcap", 1e9)
    return cfg, w
