"""Model folders for the Fekopel tests: small configurations of their own, random weights rounded to bfloat16, written as
config.json + model.safetensors."""
import json
import os

import numpy as np

import fekopel_plain as FP
from safolorn_fixture import bf16_round, rel_err, write_safetensors  # noqa: F401  (file format helpers)


def sink(heads=4, kv_heads=2, dim=10, vdim=6, window=13, scale=0.9):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if window:
        m["mask"] = {"size": window}
    return m


def gated(heads=6, kv_heads=3, dim=12, vdim=8, window=11, keep=3, scale=0.7, softcap=5.0, base=70.0, dims=8):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if window:
        m["mask"] = {"size": window, "keep_first": keep}
    if softcap:
        m["softcap"] = softcap
    if base:
        m["rot"] = {"base": base, "dims": dims}
    return m


def moe(experts=6, top=2, ff=9, groups=3, keep=2, scale=1.7, shared=14):
    f = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale}}
    if groups:
        f["router"]["groups"] = {"count": groups, "keep": keep}
    if shared:
        f["shared"] = {"ff": shared}
    return f


def attn(mixer=None, mlp=None):
    return {"type": "attention", "mixer": mixer or sink(), "mlp": mlp}


def attn2(mixer=None, mlp=None):
    return {"type": "attention_2", "mixer": mixer or gated(), "mlp": mlp}


def config(layers, vocab=59, width=38, eps=1e-5, loop=None):
    c = {"architecture": "Fekopel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


def small_config(**kw):
    """Both mixers with and without experts, one layer that sees everything; layers 1 and 2 run three times: eight layer runs."""
    kw.setdefault("loop", (1, 3, 3))
    return config([attn2(mlp=moe()), attn(mlp=moe(experts=5, top=3, groups=0, ff=7, scale=1.0, shared=0)), attn2(gated(heads=2, kv_heads=1, dim=6, vdim=10, window=0, softcap=0, base=0)),
                   attn(sink(heads=3, kv_heads=3, dim=7, vdim=4, window=5, scale=1.5), moe(experts=8, top=4, groups=4, keep=2, shared=5))], **kw)


def windowed_config(**kw):
    """No layer sees everything: pages behind the windows go back, those of the kept first tokens stay.  The loop starts at layer 0."""
    kw.setdefault("loop", (0, 2, 2))
    return config([attn2(gated(window=9, keep=6), moe(shared=0)), attn(mlp=moe()), attn2(gated(heads=2, kv_heads=2, dim=8, vdim=12, window=7, keep=2, dims=4))], **kw)


def make_model(tmp, cfg, seed=0, edit=None):
    """Writes the folder; returns (folder, weights as float64 of the bfloat16 values)."""
    W = FP.random_weights(cfg, seed)
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


def settled_tokens(cfg, W, n, seed, gap=0.04):
    """n random tokens none of whose routers faces a close call anywhere: bfloat16 rounding then changes no choice, and every row can be
    compared.  A token with one is replaced until it has none (the tokens before it do not see the change)."""
    r = np.random.default_rng(seed)
    toks = r.integers(0, cfg["vocab"], n)
    for _ in range(60 * n):
        margins = []
        FP.forward(toks, W, cfg, margins=margins)
        close = np.nonzero(np.min(margins, axis=0) < gap)[0] if margins else []
        if len(close) == 0:
            return toks
        toks[close] = r.integers(0, cfg["vocab"], len(close))
    raise AssertionError("no such tokens")


def close_enough(got, want, dtype, loose=1.0):
    """every row within rounding of the oracle, the typical one well inside"""
    got, want = np.atleast_2d(np.asarray(got, dtype=np.float64)), np.atleast_2d(np.asarray(want, dtype=np.float64))
    assert got.shape == want.shape, (got.shape, want.shape)
    e = np.sqrt(((got - want) ** 2).mean(-1)) / (np.sqrt((want ** 2).mean()) + 1e-30)
    lim = (2e-5 if dtype == "float32" else 5e-2) * loose
    if not (e.max() < lim and np.median(e) < 0.5 * lim):
        print("rows over:", np.nonzero(e >= lim)[0][:20], "worst", e.max(), "median", np.median(e))
        return False
    return True
