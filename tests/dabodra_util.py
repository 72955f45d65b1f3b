"""Helpers for the Dabodra tests: small configurations, random bf16-representable weights (optionally with one planted
query/key pair whose score stands out), a model directory written from them, and the slow oracle over the same numbers."""
from __future__ import annotations

import numpy as np

from nomanex_util import bf16_round, feed_portions, feed_whole, open_engine, rel_err, write_model_dir  # noqa: F401  (re-exported)
from oracle.dabodra_oracle import DabodraOracle, unit_rms


def moe(experts=6, top=2, count=3, keep=2, ff=10, shared=7, scale=1.3):
    return dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top, groups=dict(count=count, keep=keep), scale=scale),
                shared=dict(ff=shared) if shared else None)


def attention(heads=4, kv_heads=2, dim=6, window=9, rot_dims=4, base=100.0, scale=None, mlp="default"):
    mx = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, mask=dict(size=window), rot=dict(base=base, dims=rot_dims),
              scale=0.9 * dim ** -0.5 if scale is None else scale)
    return dict(type="attention", mixer=mx, mlp=moe() if mlp == "default" else mlp)


def delta(heads=4, kv_heads=2, dim=7, vdim=5, conv=3, mlp="default"):
    return dict(type="delta", mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv), mlp=moe() if mlp == "default" else mlp)


def make_config(layers, width=24, vocab=40, eps=1e-5):
    return dict(architecture="Dabodra", vocab=vocab, width=width, norm=dict(eps=eps), layers=layers)


def random_weights(cfg, seed=0, sink=(0.5, 1.0), a_log=(-2.0, 1.0), correction=0.3):
    """name -> float32 array whose values are exact in bfloat16."""
    rng = np.random.default_rng(seed)
    Wd = cfg["width"]
    W = {}

    def put(name, a):
        W[name] = bf16_round(np.asarray(a, dtype=np.float32))

    def mat(name, rows, cols, gain=1.0):
        put(name, rng.standard_normal((rows, cols)) * gain / np.sqrt(cols))

    def vec(name, n, mean=1.0, dev=0.2):
        put(name, mean + dev * rng.standard_normal(n))

    put("embed", rng.standard_normal((cfg["vocab"], Wd)))
    mat("head", cfg["vocab"], Wd, 2.0)
    vec("embed.norm", Wd, 0.0)
    vec("final.norm", Wd, 0.0)
    for i, ly in enumerate(cfg["layers"]):
        p, mx = "l%d." % i, ly["mixer"]
        H, G, D, Dv = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
        vec(p + "norm1", Wd, -0.1)
        if ly["type"] == "attention":
            mat(p + "mix.q", H * D, Wd, 2.0)
            mat(p + "mix.k", G * D, Wd, 2.0)
            vec(p + "mix.q.norm", H * D, 1.3)
            vec(p + "mix.k.norm", G * D, 1.3)
            vec(p + "mix.sink", H, *sink)
        else:
            for n, rows in (("q", G * D), ("k", G * D), ("v", H * Dv)):
                mat(p + "mix." + n, rows, Wd, 2.0)
                put(p + "mix." + n + ".conv", 0.6 * rng.standard_normal((rows, mx["conv"])))
            mat(p + "mix.b", H, Wd, 1.0)
            mat(p + "mix.a", H, Wd, 1.0)
            put(p + "mix.A_log", rng.uniform(*a_log, size=H))
            vec(p + "mix.dt_bias", H, -0.5, 1.0)
            vec(p + "mix.norm", Dv)
            mat(p + "mix.g", H * Dv, Wd, 2.0)
        mat(p + "mix.o", Wd, H * Dv, 2.0)
        if ly.get("mlp"):
            m = ly["mlp"]
            vec(p + "norm2", Wd, -0.1)
            mat(p + "mlp.router", m["router"]["experts"], Wd, 2.0)
            vec(p + "mlp.correction", m["router"]["experts"], 0.0, correction)
            for name, F in [("e%d" % e, m["expert"]["ff"]) for e in range(m["router"]["experts"])] + ([("shared", m["shared"]["ff"])] if m.get("shared") else []):
                mat(p + "mlp.%s.gate" % name, F, Wd, 2.0)
                mat(p + "mlp.%s.up" % name, F, Wd, 2.0)
                mat(p + "mlp.%s.down" % name, Wd, F, 2.0)
    return W


def plant_pair(cfg, W, query_token, key_token, gain=8.0):
    """Make the attention of layer 0 score key_token's key far above every other one for query_token's first query head.

    Layer 0 reads the normed embedding, so queries and keys depend on the token alone.  The key projection gets a rank-one
    term dir sel^T: sel picks out key_token's row and is orthogonal to every other token's (the vocabulary must not be
    larger than the width); dir points, inside the first key head, along the unrotated dimensions of the first query head of
    query_token, so that distance does not turn the score, and its gain makes the normed key row of key_token nearly
    parallel to it.  The same row is the value, so a query that sees it copies it."""
    mx = cfg["layers"][0]["mixer"]
    D, rot = mx["dim"], mx["rot"]["dims"]
    assert cfg["vocab"] <= cfg["width"] and rot < D
    hs = unit_rms(W["embed"].astype(np.float64), cfg["norm"]["eps"]) * (1.0 + W["embed.norm"])       # [vocab, width]
    pick = np.zeros(cfg["vocab"])
    pick[key_token] = 1.0
    sel = np.linalg.lstsq(hs, pick, rcond=None)[0]
    W["l0.mix.q.norm"][:] = 1.0
    W["l0.mix.k.norm"][:] = 1.0
    q = (W["l0.mix.q"].astype(np.float64) @ hs[query_token])[:D]
    q[:rot] = 0.0
    k = W["l0.mix.k"].astype(np.float64)
    k[:D] += gain * np.linalg.norm(k @ hs[key_token]) * np.outer(q / np.linalg.norm(q), sel)
    W["l0.mix.k"] = bf16_round(k.astype(np.float32))
    return W


def oracle_for(cfg, W):
    return DabodraOracle(cfg, W)
