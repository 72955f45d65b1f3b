"""The Soselix oracle's mechanisms against independent closed forms (CPU), the planted-pair construction the GPU tests
rely on, and the host-side configuration checks, which run before any device is touched."""
import json

import numpy as np
import pytest

from oracle import soselix_oracle as O
from soselix_util import hgrn2, latent, make_config, mamba2, oracle_for, plant_pair, random_weights, rel_err, write_model_dir


def params(cfg, seed, layer=0, part="mix."):
    return O.sub({k: v.astype(np.float64) for k, v in random_weights(cfg, seed=seed).items()}, "l%d.%s" % (layer, part))


def test_rotation_pairs_a_dimension_with_the_one_half_the_span_further():
    rng = np.random.default_rng(0)
    rot = dict(dims=6, base=50.0)
    q, k = rng.standard_normal((1, 6)), rng.standard_normal((1, 6))
    a = (O.rotate_half(q, 11, rot) @ O.rotate_half(k, 4, rot).T).item()
    b = (O.rotate_half(q, 27, rot) @ O.rotate_half(k, 20, rot).T).item()
    assert abs(a - b) < 1e-9                                        # relative
    r = O.rotate_half(np.array([[1.0, 0.0, 0.0, 0.0]]), 1, dict(dims=4, base=50.0))
    assert np.allclose(r, [[np.cos(1.0), 0.0, np.sin(1.0), 0.0]])    # entry 0 turns with entry 2, at frequency 1
    r = O.rotate_half(np.array([[0.0, 1.0, 0.0, 0.0]]), 2, dict(dims=4, base=49.0))
    assert np.allclose(r, [[0.0, np.cos(2.0 / 7.0), 0.0, np.sin(2.0 / 7.0)]])    # entry 1 with entry 3, at base^(-2/4)


def test_sink_counts_once_in_the_denominator_and_has_no_value():
    s = np.array([0.3, -1.0, 2.0])
    w = O.sink_softmax(s, 0.5)
    full = np.exp(np.append(s, 0.5))
    assert np.allclose(w, (full / full.sum())[:3]) and w.sum() < 1.0
    assert np.allclose(O.sink_softmax(s, -1e9), np.exp(s) / np.exp(s).sum())
    assert O.sink_softmax(np.array([0.0]), 800.0)[0] == 0.0           # a huge sink takes everything, without overflow


def test_carried_convolution_equals_the_direct_sum():
    rng = np.random.default_rng(1)
    w, b, u = rng.standard_normal((3, 4)), rng.standard_normal(3), rng.standard_normal((9, 3))
    cv = O.CarriedConv(w, b)
    got = np.stack([cv.step(x) for x in u])
    for t in range(9):
        want = b + sum(w[:, j] * u[t - 3 + j] for j in range(4) if t - 3 + j >= 0)    # the last tap is the token's own
        assert np.abs(got[t] - want).max() < 1e-12


def dense_attention(P, Pkv, mx, hs, eps=1e-5):
    """All positions at once, keys and values rebuilt per head from the latents that Pkv makes."""
    T, H, D, R, Dv, C = len(hs[0]), mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"], mx["kv_rank"]
    rms = lambda v: np.sqrt((v * v).mean(-1, keepdims=True) + eps)
    cq = hs[0] @ P["dq"].T
    q = ((cq / rms(cq) * P["dq.norm"]) @ P["uq"].T).reshape(T, H, D + R)
    d = hs[1] @ Pkv["dkv"].T
    c = d[:, :C] / rms(d[:, :C]) * Pkv["dkv.norm"]
    kr = np.stack([O.rotate_half(d[t:t + 1, C:], t, mx["rot"])[0] for t in range(T)])
    qr = np.stack([O.rotate_half(q[t, :, D:], t, mx["rot"]) for t in range(T)])
    k, v = (c @ P["uk"].T).reshape(T, H, D), (c @ P["uv"].T).reshape(T, H, Dv)
    out = np.zeros((T, H, Dv))
    for h in range(H):
        s = (q[:, h, :D] @ k[:, h].T + qr[:, h] @ kr.T) * mx["scale"]
        e = np.exp(np.where(np.tril(np.ones((T, T), bool)), s, -np.inf))
        out[:, h] = e / (e.sum(-1, keepdims=True) + np.exp(P["sink"][h])) @ v[:, h] / (1.0 + np.exp(-hs[0] @ P["g"][h]))[:, None]
    return out.reshape(T, -1) @ P["o"].T


def test_latent_attention_equals_dense_causal_attention_over_rebuilt_keys():
    cfg = make_config([latent(mlp=None)], width=10)
    P, mx = params(cfg, 1), cfg["layers"][0]["mixer"]
    hs = np.random.default_rng(2).standard_normal((11, 10))
    at = O.LatentAttention(P, mx, 1e-5)
    got = np.stack([at.step(h) for h in hs])
    assert np.abs(got - dense_attention(P, P, mx, (hs, hs))).max() < 1e-10


def test_a_layer_reads_another_layers_latents_with_its_own_projections():
    cfg = make_config([latent(mlp=None), latent(heads=2, dim=3, vdim=4, q_rank=5, kv_from=0, mlp=None)], width=10)
    P0, P1 = params(cfg, 3), params(cfg, 3, 1)
    assert "dkv" not in P1
    m0, m1 = cfg["layers"][0]["mixer"], cfg["layers"][1]["mixer"]
    rng = np.random.default_rng(4)
    h0, h1 = rng.standard_normal((9, 10)), rng.standard_normal((9, 10))
    a = O.LatentAttention(P0, m0, 1e-5)
    b = O.LatentAttention(P1, m1, 1e-5, a.cache)
    got = []
    for t in range(9):
        a.step(h0[t])
        got.append(b.step(h1[t]))
    assert np.abs(np.stack(got) - dense_attention(P1, P0, m1, (h1, h0))).max() < 1e-10


def test_forget_gate_and_its_complement():
    z = np.array([-40.0, -1.0, 0.0, 3.0, 40.0])
    f, w = O.forget_gate(z, np.full(5, 0.25))
    assert np.allclose(f + w, 1.0) and np.all(f >= 0.25) and f[4] == 1.0 and w[4] > 0.0       # the complement survives where f rounds to 1
    assert np.allclose(f[1], 0.25 + 0.75 / (1.0 + np.e))


def test_hgrn2_equals_the_unrolled_sum():
    cfg = make_config([hgrn2(heads=2, dim=3, vdim=4, mlp=None)], width=6)
    P = params(cfg, 5)
    hs = np.random.default_rng(6).standard_normal((7, 6))
    mm = O.Hgrn2(P, cfg["layers"][0]["mixer"], 1e-5)
    got = np.stack([mm.step(h) for h in hs])
    q = hs @ P["q"].T
    q = (q / (1.0 + np.exp(-q))).reshape(7, 2, 3)
    v = (hs @ P["v"].T).reshape(7, 2, 4)
    f = (P["lower"] + (1.0 - P["lower"]) / (1.0 + np.exp(-(hs @ P["f"].T + P["f.b"])))).reshape(7, 2, 3)
    for t in range(7):
        o = np.zeros((2, 4))
        for h in range(2):
            # token j's write (1 - f_j), decayed by every later f, read by q_t
            o[h] = sum(((1.0 - f[j, h]) * np.prod(f[j + 1:t + 1, h], axis=0) * q[t, h]).sum() * v[j, h] for j in range(t + 1))
        o = o / np.sqrt((o * o).mean(-1, keepdims=True) + 1e-5) * P["norm"]
        assert np.abs(got[t] - P["o"] @ o.reshape(-1)).max() < 1e-10


def test_mamba2_equals_the_unrolled_sum():
    cfg = make_config([mamba2(heads=4, vdim=3, state=2, groups=2, norm_groups=3, conv=2, mlp=None)], width=6)
    P = params(cfg, 7)
    hs = np.random.default_rng(8).standard_normal((6, 6))
    mm = O.Mamba2(P, cfg["layers"][0]["mixer"], 1e-5)
    got = np.stack([mm.step(h) for h in hs])
    u = hs @ P["in"].T
    z, xbc, dt = u[:, :12], u[:, 12:32], u[:, 32:]
    a = np.stack([P["conv.b"] + P["conv"][:, 1] * xbc[t] + (P["conv"][:, 0] * xbc[t - 1] if t else 0.0) for t in range(6)])
    a = a / (1.0 + np.exp(-a))
    x, B, C = a[:, :12].reshape(6, 4, 3), a[:, 12:16].reshape(6, 2, 2), a[:, 16:].reshape(6, 2, 2)
    d = np.log1p(np.exp(dt + P["dt_bias"]))
    for t in range(6):
        y = np.zeros((4, 3))
        for h in range(4):
            g = 0 if h < 2 else 1                       # heads 0, 1 read group 0
            y[h] = sum(np.exp(-np.exp(P["A_log"][h]) * d[j + 1:t + 1, h].sum()) * d[j, h] * (B[j, g] @ C[t, g]) * x[j, h] for j in range(t + 1))
            y[h] += P["D"][h] * x[t, h]
        y = (y.reshape(-1) * z[t] / (1.0 + np.exp(-z[t]))).reshape(3, 4)      # the gate first, then the norm of every third
        y = (y / np.sqrt((y * y).mean(-1, keepdims=True) + 1e-5)).reshape(-1) * P["norm"]
        assert np.abs(got[t] - P["o"] @ y).max() < 1e-10


def test_xielu_pieces_meet_and_follow_their_formulas():
    p, q = 0.3, -0.7
    sp, sq = np.log1p(np.exp(p)), np.log1p(np.exp(q))
    assert np.allclose(O.xielu(np.array([2.0]), p, q), sp * 4.0 + 1.0)
    assert np.allclose(O.xielu(np.array([-2.0]), p, q), (0.5 + sq) * (np.exp(-2.0) + 1.0) - 1.0)
    e = 1e-6
    lo, mid, hi = O.xielu(np.array([-e, 0.0, e]), p, q)
    assert mid == 0.0 and abs((hi - lo) / (2 * e) - 0.5) < 1e-5             # value 0 and slope 1/2 at the joint
    P = params(make_config([hgrn2()], width=6), 9, part="mlp.")
    h = np.random.default_rng(1).standard_normal(6)
    z = P["up"] @ h + P["up.b"]
    assert np.allclose(O.dense_ff(P, h), P["down"] @ O.xielu(z, *P["act"]) + P["down.b"])


def test_residual_multiplier_and_embedding_scale():
    cfg = make_config([hgrn2()], mult=0.25, embed=3.0)
    W = random_weights(cfg, seed=11)
    o = oracle_for(cfg, W)
    lg, ly = o.forward([5], return_layers=True)
    x = W["embed"][5].astype(np.float64) * 3.0
    x = x + 0.25 * O.Hgrn2(O.sub(o.W, "l0.mix."), cfg["layers"][0]["mixer"], 1e-5).step(o.norm("l0.norm1", x))
    x = x + 0.25 * O.dense_ff(O.sub(o.W, "l0.mlp."), o.norm("l0.norm2", x))
    assert np.abs(ly[0, 0] - x).max() < 1e-12
    assert np.abs(lg[0] - o.W["head"] @ (x / np.sqrt((x * x).mean() + 1e-5) * float(W["final.norm"]))).max() < 1e-12


def test_planted_pair_makes_one_key_decide():
    cfg = make_config([latent(heads=2, dim=12, vdim=10, kv_rank=16, q_rank=20, scale=3.0, mlp=None)], width=48, vocab=40)
    o = oracle_for(cfg, plant_pair(cfg, random_weights(cfg, seed=31, sink=(3.0, 0.2)), 7, 11))
    a = np.random.default_rng(1).integers(12, 40, size=60).tolist()
    a[55] = 7
    b = list(a)
    a[3] = 11
    assert rel_err(o.forward(a)[55:56], o.forward(b)[55:56])[0] > 0.3


def test_config_errors_come_before_any_device_work(tmp_path):
    from kubeai_b200 import B200Error
    from kubeai_b200.engine import Engine, default_config
    cfg = make_config([latent(), hgrn2(), mamba2(), latent(kv_from=0)])
    W = random_weights(cfg)
    lim = default_config(manual_step=1)
    mx = lambda c, i: c["layers"][i]["mixer"]
    for i, (edit, msg) in enumerate([
            (lambda c: c["layers"][0].update(type="rwkv"), "unknown mixer"),
            (lambda c: mx(c, 0).pop("kv_rank"), "kv_rank"),
            (lambda c: mx(c, 0)["rot"].update(dims=6), "rot"),
            (lambda c: mx(c, 3).update(kv_from=3), "kv_from"),
            (lambda c: mx(c, 3).update(kv_from=1), "kv_from"),
            (lambda c: mx(c, 3).update(kv_rank=8), "kv_rank, rot_dim and rotation"),
            (lambda c: mx(c, 3)["rot"].update(base=9.0), "kv_rank, rot_dim and rotation"),
            (lambda c: mx(c, 2).update(groups=3), "groups"),
            (lambda c: mx(c, 2).update(norm_groups=7), "norm_groups"),
            (lambda c: mx(c, 1).update(dim=0), "dim"),
            (lambda c: c["layers"][1]["mlp"].update(kind="moe"), "mlp.kind"),
            (lambda c: c.pop("width"), "width")]):
        bad = json.loads(json.dumps(cfg))
        edit(bad)
        with pytest.raises(B200Error, match=msg):
            Engine(lim, write_model_dir(tmp_path / ("b%d" % i), bad, W), dtype="float32")
