"""Tiny Gezavik configurations for the tests: both mixers and both feed-forwards, layers in several orders, with and without
the keys a layer may go without (window, shared expert, identities, feed-forward), and sizes chosen so that nothing that
could be confused is equal (heads and groups, head size and state, the norm's parts and the heads, plain, rotated and value
dims, query and key latents, experts and router outputs) or happens to be 1 by accident.  The recurrences' decay rates and
step sizes are moved so that a state lives for tens of tokens, the convolutions' taps and the routers' rows are made larger
than the other weights, so that neither is flat."""
from __future__ import annotations

import json
import os

import numpy as np
import torch

import helpers


def mamba(heads, vdim, state, groups, conv, norm_groups):
    return {"conv": conv, "groups": groups, "heads": heads, "norm_groups": norm_groups, "state": state, "vdim": vdim}


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, base, window=None):
    m = {"dim": dim, "heads": heads, "kv_rank": kv_rank, "q_rank": q_rank, "rot": {"base": base, "dims": rot_dim}, "rot_dim": rot_dim,
         "scale": scale, "vdim": vdim}
    if window:
        m["mask"] = {"size": window}
    return m


def dense(ff):
    return {"ff": ff, "kind": "dense"}


def moe(ff, limit, experts, identity, top, shared=None):
    m = {"expert": {"ff": ff, "limit": limit}, "kind": "moe", "router": {"experts": experts, "identity": identity, "top": top}}
    if shared:
        m["shared"] = {"ff": shared[0], "limit": shared[1]}
    return m


def layer(kind, mixer, mlp):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


def config(width, vocab, eps, mult, layers, std):
    return {"architecture": "Gezavik", "width": width, "vocab": vocab, "norm": {"eps": eps}, "residual_mult": mult, "layers": layers,
            "initializer_range": std}


CONFIGS = {
    # cache rows of 16 numbers (the tensor-core decode kernels' smallest head), a window shorter than a page run; the norm's
    # parts cut across heads; a layer without feed-forward; no shared expert; a query latent that no 16-byte load divides
    "A": config(48, 131, 1e-6, 0.45, [
        layer("mamba2", mamba(6, 8, 16, 3, 3, 4), moe(24, 0.8, 5, 1, 2)),
        layer("latent_attention", latent(3, 8, 4, 12, 20, 12, 0.5, 900.0, window=7), dense(72)),
        layer("mamba2", mamba(2, 24, 8, 1, 2, 2), None),
        layer("latent_attention", latent(4, 10, 6, 8, 24, 10, 0.45, 5000.0, window=19), moe(16, 1.5, 4, 3, 3, (40, 0.6))),
    ], 0.12),
    # a cache row of 26 numbers (no tensor-core kernel takes it); three groups of two heads over states of 24; more identities
    # than are chosen; full attention in one layer
    "B": config(64, 200, 1e-5, 0.7, [
        layer("latent_attention", latent(2, 16, 6, 24, 32, 20, 0.35, 10000.0, window=33), dense(96)),
        layer("mamba2", mamba(6, 16, 24, 3, 4, 6), moe(24, 1.0, 6, 4, 4, (32, 1.2))),
        layer("mamba2", mamba(4, 8, 40, 2, 5, 1), dense(40)),
        layer("latent_attention", latent(5, 8, 8, 16, 40, 24, 0.4, 700.0), moe(32, 2.0, 3, 1, 1, (24, 0.9))),
    ], 0.1),
    # the tensor-core kernels' sizes: cache rows of 64 and of 144 numbers, states of 128 and 64 with value heads of 64 and 40
    # (the chunked walk with both of its block widths), expert sizes of the grouped tcgen05 product
    "C": config(128, 300, 1e-5, 0.35, [
        layer("mamba2", mamba(4, 64, 128, 2, 4, 2), moe(40, 1.2, 6, 2, 3, (64, 0.8))),
        layer("latent_attention", latent(8, 32, 16, 48, 72, 48, 0.3, 20000.0, window=37), dense(320)),
        layer("mamba2", mamba(6, 40, 64, 1, 3, 8), dense(160)),
        layer("latent_attention", latent(4, 16, 16, 40, 56, 128, 0.35, 100000.0), moe(48, 0.9, 8, 1, 2)),
    ], 0.08),
    # sizes that no vector load divides: a width of 8 * 5, an odd vocabulary, value heads of 5 over states of 10, one tap, a
    # latent of 9 and two rotated dims; every output of the router chosen; no identities in one layer
    "D": config(40, 103, 1e-6, 1.0, [
        layer("mamba2", mamba(3, 5, 10, 3, 1, 5), moe(12, 0.7, 2, 1, 3, (20, 1.1))),
        layer("latent_attention", latent(3, 7, 2, 5, 11, 9, 0.6, 100.0, window=2), None),
        layer("mamba2", mamba(1, 21, 34, 1, 2, 3), moe(20, 1.3, 6, 0, 1)),
        layer("latent_attention", latent(1, 5, 4, 13, 7, 6, 0.6, 3000.0, window=1), dense(30)),
    ], 0.15),
}
SEEDS = {"A": 61, "B": 62, "C": 63, "D": 64}
# tensors whose names end so: value * factor + shift
SHARPEN = {".conv": (6.0, 0.0), ".conv.b": (2.0, 0.0), ".A_log": (4.0, -2.5), ".dt_bias": (4.0, -0.5), ".router": (3.0, 0.0),
           ".correction": (0.4, 0.0), ".mix.D": (3.0, 0.3)}


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
    d = os.path.join(str(tmpdir), f"gezavik_{which}_{str(dtype).split('.')[-1]}")
    os.makedirs(d, exist_ok=True)
    with open(os.path.join(d, "config.json"), "w", encoding="utf-8") as f:
        json.dump(cfg.to_dict(), f, indent=1)
    save_file(tensors, os.path.join(d, "model.safetensors"))
    return d


def prompts(which: str, rng: np.random.Generator, lengths):
    return [rng.integers(0, CONFIGS[which]["vocab"], n).tolist() for n in lengths]


def routed_prefixes(cfg: dict):
    """The tensor prefixes of the routed feed-forwards, in running order."""
    return [f"l{i}.mlp." for i, e in enumerate(cfg["layers"]) if e.get("mlp") and e["mlp"]["kind"] == "moe"]


load_plain = helpers.load_plain
