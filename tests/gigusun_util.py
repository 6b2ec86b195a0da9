"""Small Gigusun configurations for the tests: sizes that are deliberately unequal and odd."""
from __future__ import annotations

import importlib

import numpy as np


def attention(heads=6, kv_heads=2, dim=40, vdim=24, size=13, keep_first=3, softcap=20.0, scale=None, ff=72):
    return {"type": "attention", "mlp": None if ff is None else {"kind": "dense", "ff": ff},
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "softcap": softcap,
                      "scale": dim ** -0.5 if scale is None else scale, "mask": {"size": size, "keep_first": keep_first}}}


def gla(heads=3, dim=20, vdim=36, tau=7.0, ff=72):
    return {"type": "gla", "mlp": None if ff is None else {"kind": "dense", "ff": ff},
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}}


def delta(heads=4, kv_heads=2, dim=28, vdim=20, conv=4, ff=72):
    return {"type": "delta", "mlp": None if ff is None else {"kind": "dense", "ff": ff},
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def artifacts(pkg):
    return importlib.import_module(f"{pkg.__name__}.artifact")


def make_model(pkg, directory, layers, seed=1, *, vocab=300, width=56, max_positions=512, eps=1e-5, decay_rank=6,
               edit=None):
    """Writes a random model; returns (directory, config, float64 weights for the oracle).  `edit(weights)` may
    change the F32 weights in place (values are rounded to BF16 again before they are written)."""
    art = artifacts(pkg)
    config = art.gigusun_config(layers, vocab=vocab, width=width, max_positions=max_positions, eps=eps)
    weights = art.decoder_weights(config, seed, decay_rank)
    if edit is not None:
        edit(weights)
        for name, values in weights.items():
            bits = np.frombuffer(art._bf16_bytes(values), np.uint16).astype(np.uint32) << 16
            weights[name] = bits.view(np.float32).reshape(values.shape)
    art.write_decoder(directory, config, weights)
    return directory, config, {name: values.astype(np.float64) for name, values in weights.items()}
