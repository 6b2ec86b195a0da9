"""Small Kikepel configurations for the tests: sizes that are deliberately unequal and odd."""
from __future__ import annotations

import importlib

import numpy as np


def dense(ff=88):
    return {"kind": "dense", "ff": ff}


def moe(experts=6, top=2, ff=40, limit=0.8):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def latent(heads=5, dim=24, vdim=40, q_rank=56, kv_rank=72, size=21, scale=None, sink=True, mlp=None):
    return {"type": "latent_attention" if sink else "latent_attention_2", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                      "scale": dim ** -0.5 if scale is None else scale, "mask": {"size": size}}}


def artifacts(pkg):
    return importlib.import_module(f"{pkg.__name__}.artifact")


def round_bf16(art, values):
    bits = np.frombuffer(art._bf16_bytes(values), np.uint16).astype(np.uint32) << 16
    return bits.view(np.float32).reshape(values.shape)


def make_model(pkg, directory, layers, seed=1, *, vocab=300, width=72, logit_scale=1.7, logit_softcap=9.0, eps=1e-4,
               edit=None):
    """Writes a random model; returns (directory, config, float64 weights for the oracle).  `edit(weights)` may
    change the F32 weights in place (values are rounded to BF16 again before they are written)."""
    art = artifacts(pkg)
    config = art.kikepel_config(layers, vocab=vocab, width=width, logit_scale=logit_scale, logit_softcap=logit_softcap,
                                eps=eps)
    weights = art.decoder_weights(config, seed)
    if edit is not None:
        edit(weights)
        weights = {name: round_bf16(art, values) for name, values in weights.items()}
    art.write_decoder(directory, config, weights)
    return directory, config, {name: values.astype(np.float64) for name, values in weights.items()}
