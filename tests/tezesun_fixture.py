"""Model folders for the Tezesun tests: small configurations of their own, random weights rounded to bfloat16, written as
config.json + model.safetensors."""
import json
import os

import numpy as np

import tezesun_plain as TP
from safolorn_fixture import bf16_round, close_enough, rel_err, write_safetensors  # noqa: F401  (file format helpers)


def attention(heads=4, kv_heads=2, dim=10, vdim=6, window=13, keep=3, scale=0.3, softcap=5.0, diff=0.3, base=50.0, dims=8, scaling=True):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff}
    if window:
        m["mask"] = {"size": window, "keep_first": keep}
    if softcap:
        m["softcap"] = softcap
    if base:
        m["rot"] = {"base": base, "dims": dim if dims is None else dims}
        if scaling:  # with base 50 and 8 dimensions: the ramp starts at frequency 0 and ends inside the others
            m["rot"]["scaling"] = {"factor": 3.0, "original": 64, "fast": 8.0, "slow": 1.0}
    return m


def latent(heads=3, dim=7, rot_dim=4, vdim=5, kv_rank=9, q_rank=11, scale=0.35, base=200.0):
    return {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": scale,
            "rot": {"base": base, "dims": rot_dim}}


def rglru(width=24, blocks=3, conv=3):
    return {"width": width, "blocks": blocks, "conv": conv}


def layer(kind, mixer, ff=0):
    return {"type": kind, "mixer": mixer, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(layers, vocab=61, width=36, eps=1e-5, logit_scale=0.7):
    return {"architecture": "Tezesun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": logit_scale, "layers": layers}


def small_config(**kw):
    """Every mixer with and without a feed-forward."""
    return config([layer("rglru", rglru(), 20), layer("attention", attention(), 17), layer("latent_attention", latent(), 28),
                   layer("attention", attention(heads=3, kv_heads=3, dim=6, vdim=10, window=5, keep=2, softcap=0, base=0, diff=0.6)),
                   layer("rglru", rglru(width=14, blocks=1, conv=5)), layer("latent_attention", latent(heads=2, dim=4, rot_dim=6, vdim=8, kv_rank=6, q_rank=5))], **kw)


def windowed_config(**kw):
    """No layer sees everything: pages behind the windows go back, those of the kept first tokens stay."""
    return config([layer("attention", attention(), 17), layer("rglru", rglru(), 12),
                   layer("attention", attention(heads=2, kv_heads=1, dim=8, vdim=8, window=7, keep=6, scaling=False), 9)], **kw)


def make_model(tmp, cfg, seed=0, edit=None):
    """Writes the folder; returns (folder, weights as float64 of the bfloat16 values)."""
    W = TP.random_weights(cfg, seed)
    if edit:
        edit(W)
    out, vals = {}, {}
    for k, v in W.items():
        vals[k], codes = bf16_round(v)
        out[k] = (codes, np.shape(v))
    os.makedirs(tmp, exist_ok=True)
    with open(os.path.join(tmp, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(tmp, "model.safetensors"), out, misalign=True)
    return tmp, vals
