"""Helpers for the Soselix tests: small configurations, random bf16-representable weights (optionally with one planted
query/key pair whose score stands out), a model directory written from them, and the slow oracle over the same numbers."""
from __future__ import annotations

import numpy as np

from nomanex_util import bf16_round, feed_portions, feed_whole, open_engine, rel_err, write_model_dir  # noqa: F401  (re-exported)
from oracle.soselix_oracle import SoselixOracle, unit_rms


def latent(heads=3, dim=6, rot_dim=4, vdim=5, kv_rank=10, q_rank=9, base=100.0, scale=None, kv_from=None, mlp="default"):
    mx = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, q_rank=q_rank, rot=dict(base=base, dims=rot_dim),
              scale=0.9 * (dim + rot_dim) ** -0.5 if scale is None else scale)
    if kv_from is not None:
        mx["kv_from"] = kv_from
    return dict(type="latent_attention", mixer=mx, mlp=dense() if mlp == "default" else mlp)


def hgrn2(heads=2, dim=7, vdim=5, mlp="default"):
    return dict(type="hgrn2", mixer=dict(heads=heads, dim=dim, vdim=vdim), mlp=dense() if mlp == "default" else mlp)


def mamba2(heads=4, vdim=6, state=5, groups=2, norm_groups=3, conv=3, mlp="default"):
    return dict(type="mamba2", mixer=dict(heads=heads, vdim=vdim, state=state, groups=groups, norm_groups=norm_groups, conv=conv),
                mlp=dense() if mlp == "default" else mlp)


def dense(ff=18):
    return dict(kind="dense", ff=ff)


def make_config(layers, width=24, vocab=40, eps=1e-5, mult=0.6, embed=1.7):
    return dict(architecture="Soselix", vocab=vocab, width=width, norm=dict(eps=eps), residual_mult=mult, embedding=dict(scale=embed), layers=layers)


def random_weights(cfg, seed=0, sink=(0.5, 1.0), lower=(0.0, 0.9), q_gain=1.0):
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

    def one(name):
        put(name, 1.0 + 0.2 * rng.standard_normal())

    put("embed", rng.standard_normal((cfg["vocab"], Wd)))
    mat("head", cfg["vocab"], Wd, 2.0)
    one("final.norm")
    for i, ly in enumerate(cfg["layers"]):
        p, mx = "l%d." % i, ly["mixer"]
        H, Dv = mx["heads"], mx["vdim"]
        one(p + "norm1")
        if ly["type"] == "latent_attention":
            D, R, C, Q = mx["dim"], mx["rot_dim"], mx["kv_rank"], mx["q_rank"]
            mat(p + "mix.dq", Q, Wd, 2.0)
            vec(p + "mix.dq.norm", Q)
            mat(p + "mix.uq", H * (D + R), Q, 3.0 * q_gain)
            if mx.get("kv_from") is None:
                mat(p + "mix.dkv", C + R, Wd, 2.0)
                vec(p + "mix.dkv.norm", C)
            mat(p + "mix.uk", H * D, C, 2.0)
            mat(p + "mix.uv", H * Dv, C, 2.0)
            vec(p + "mix.sink", H, *sink)
            mat(p + "mix.g", H, Wd, 2.0)
        elif ly["type"] == "hgrn2":
            D = mx["dim"]
            mat(p + "mix.q", H * D, Wd, 2.0)
            mat(p + "mix.f", H * D, Wd, 2.0)
            vec(p + "mix.f.b", H * D, 1.0, 1.0)
            put(p + "mix.lower", rng.uniform(*lower, size=H * D))
            mat(p + "mix.v", H * Dv, Wd, 2.0)
            vec(p + "mix.norm", Dv)
        else:
            ch = H * Dv + 2 * mx["groups"] * mx["state"]
            mat(p + "mix.in", H * Dv + ch + H, Wd, 2.0)
            put(p + "mix.conv", 0.6 * rng.standard_normal((ch, mx["conv"])))
            vec(p + "mix.conv.b", ch, 0.0, 0.2)
            vec(p + "mix.dt_bias", H, -1.0, 1.0)
            put(p + "mix.A_log", np.log(rng.uniform(0.05, 4.0, size=H)))
            vec(p + "mix.D", H)
            vec(p + "mix.norm", H * Dv)
        mat(p + "mix.o", Wd, H * Dv, 2.0)
        if ly.get("mlp"):
            F = ly["mlp"]["ff"]
            one(p + "norm2")
            mat(p + "mlp.up", F, Wd, 2.0)
            vec(p + "mlp.up.b", F, 0.0, 0.4)
            mat(p + "mlp.down", Wd, F, 1.0)
            vec(p + "mlp.down.b", Wd, 0.0, 0.4)
            vec(p + "mlp.act", 2, 0.0, 1.0)
    return W


def plant_pair(cfg, W, query_token, key_token, gain=8.0):
    """Make the attention of layer 0 score key_token's latent far above every other one for query_token's queries.

    Layer 0 sees nothing but the token, so a token's latent depends on the token alone.  The latent projection gets a
    rank-one term dir sel^T: sel picks out key_token's normed input and is orthogonal to every other token's (the
    vocabulary must not be larger than the width); dir points, in latent space, along the first head's absorbed query
    W_uk^T q of query_token, so the normed latent of key_token is nearly parallel to it and no other one is.  The rotated
    parts are switched off, so that distance alone changes nothing.  With a sharp softmax a query_token position then
    copies the values of the visible key_token positions, and its logits change visibly when such a position is gone."""
    mx = cfg["layers"][0]["mixer"]
    H, D, R, C = mx["heads"], mx["dim"], mx["rot_dim"], mx["kv_rank"]
    assert cfg["vocab"] <= cfg["width"]
    eps = cfg["norm"]["eps"]
    hs = unit_rms(W["embed"].astype(np.float64) * cfg["embedding"]["scale"], eps) * float(W["l0.norm1"])      # [vocab, width]
    pick = np.zeros(cfg["vocab"])
    pick[key_token] = 1.0
    sel = np.linalg.lstsq(hs, pick, rcond=None)[0]
    cq = unit_rms(W["l0.mix.dq"].astype(np.float64) @ hs[query_token], eps) * W["l0.mix.dq.norm"]
    q = (W["l0.mix.uq"].astype(np.float64) @ cq).reshape(H, D + R)[0, :D]
    d = W["l0.mix.uk"].astype(np.float64).reshape(H, D, C)[0].T @ q
    dkv = W["l0.mix.dkv"].astype(np.float64)
    dkv[:C] += gain * np.linalg.norm(dkv[:C] @ hs[key_token]) * np.outer(d / np.linalg.norm(d), sel)
    dkv[C:] = 0.0
    W["l0.mix.dkv"] = bf16_round(dkv.astype(np.float32))
    W["l0.mix.dkv.norm"][:] = 1.0
    return W


def oracle_for(cfg, W):
    return SoselixOracle(cfg, W)
