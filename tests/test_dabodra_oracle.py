"""The Dabodra oracle's mechanisms against independent closed forms (CPU), the planted-pair construction the GPU tests
rely on, and the host-side configuration checks, which run before any device is touched."""
import json

import numpy as np
import pytest

from dabodra_util import attention, delta, make_config, moe, oracle_for, plant_pair, random_weights, rel_err, write_model_dir
from oracle import dabodra_oracle as O


def params(cfg, seed, layer=0, part="mix."):
    return O.sub({k: v.astype(np.float64) for k, v in random_weights(cfg, seed=seed).items()}, "l%d.%s" % (layer, part))


def test_rotation_pairs_neighbouring_dimensions():
    rng = np.random.default_rng(0)
    rot = dict(dims=6, base=50.0)
    q, k = rng.standard_normal((1, 8)), rng.standard_normal((1, 8))
    a = (O.rotate_pairs(q, 11, rot) @ O.rotate_pairs(k, 4, rot).T).item()
    b = (O.rotate_pairs(q, 27, rot) @ O.rotate_pairs(k, 20, rot).T).item()
    assert abs(a - b) < 1e-9                                        # relative
    assert np.array_equal(O.rotate_pairs(q, 11, rot)[:, 6:], q[:, 6:])
    r = O.rotate_pairs(np.array([[1.0, 0.0, 0.0, 0.0]]), 1, dict(dims=4, base=50.0))
    assert np.allclose(r, [[np.cos(1.0), np.sin(1.0), 0.0, 0.0]])    # entry 0 turns with entry 1, at frequency 1
    r = O.rotate_pairs(np.array([[0.0, 0.0, 1.0, 0.0]]), 2, dict(dims=4, base=49.0))
    assert np.allclose(r, [[0.0, 0.0, np.cos(2.0 / 7.0), np.sin(2.0 / 7.0)]])    # entry 2 with entry 3, at base^(-2/4)


def test_window_attention_equals_a_masked_dense_one():
    """All positions at once: a band of `size` keys, the sink as one more column without a value, rows normed whole."""
    cfg = make_config([attention(window=5, mlp=None)], width=10)
    P, mx = params(cfg, 1), cfg["layers"][0]["mixer"]
    H, G, D, T = mx["heads"], mx["kv_heads"], mx["dim"], 14
    hs = np.random.default_rng(2).standard_normal((T, 10))
    at = O.WindowAttention(P, mx, 1e-5)
    got = np.stack([at.step(h) for h in hs])
    rms = lambda v: np.sqrt((v * v).mean(-1, keepdims=True) + 1e-5)
    q, k = hs @ P["q"].T, hs @ P["k"].T
    v = k.reshape(T, G, D)
    qr = (q / rms(q) * P["q.norm"]).reshape(T, H, D)
    kr = (k / rms(k) * P["k.norm"]).reshape(T, G, D)
    qr = np.stack([O.rotate_pairs(qr[t], t, mx["rot"]) for t in range(T)])
    kr = np.stack([O.rotate_pairs(kr[t], t, mx["rot"]) for t in range(T)])
    i, j = np.arange(T)[:, None], np.arange(T)[None]
    seen = (j <= i) & (i - j < 5)
    out = np.zeros((T, H, D))
    for h in range(H):
        e = np.exp(np.where(seen, qr[:, h] @ kr[:, h * G // H].T * mx["scale"], -np.inf))
        out[:, h] = e / (e.sum(-1, keepdims=True) + np.exp(P["sink"][h])) @ v[:, h * G // H]
    assert np.abs(got - out.reshape(T, -1) @ P["o"].T).max() < 1e-10


def test_sink_counts_once_in_the_denominator_and_has_no_value():
    s = np.array([0.3, -1.0, 2.0])
    w = O.sink_softmax(s, 0.5)
    full = np.exp(np.append(s, 0.5))
    assert np.allclose(w, (full / full.sum())[:3]) and w.sum() < 1.0
    assert O.sink_softmax(np.array([0.0]), 800.0)[0] == 0.0           # a huge sink takes everything, without overflow


def test_carried_convolution_equals_the_direct_sum():
    rng = np.random.default_rng(1)
    w, u = rng.standard_normal((3, 4)), rng.standard_normal((9, 3))
    cv = O.CarriedConv(w)
    got = np.stack([cv.step(x) for x in u])
    for t in range(9):
        want = sum(w[:, j] * u[t - 3 + j] for j in range(4) if t - 3 + j >= 0)    # the last tap is the token's own
        assert np.abs(got[t] - want).max() < 1e-12


def test_delta_update_solves_the_unrolled_triangular_system():
    """With c the running product of the decays: u_t = beta_t (v_t - c_t S0^T k_t - sum_{j<t} (c_t / c_j)(k_j . k_t) u_j), a
    triangular system in u, and o_t = c_t S0^T q_t + sum_{j<=t} (c_t / c_j)(k_j . q_t) u_j."""
    rng = np.random.default_rng(3)
    T, D, Dv = 12, 5, 4
    q, k, v = rng.standard_normal((T, D)), O.unit_length(rng.standard_normal((T, D))), rng.standard_normal((T, Dv))
    g, beta = rng.uniform(0.3, 1.0, T), rng.uniform(0.0, 1.0, T)
    S0 = rng.standard_normal((D, Dv))
    c = np.cumprod(g)
    ratio = c[:, None] / c[None]
    A = np.tril(ratio * (k @ k.T), -1) * beta[:, None]
    u = np.linalg.solve(np.eye(T) + A, beta[:, None] * (v - c[:, None] * (k @ S0)))
    want = c[:, None] * (q @ S0) + np.tril(ratio * (q @ k.T)) @ u
    S, got = S0, []
    for t in range(T):
        S, o = O.delta_update(S, g[t], beta[t], q[t], k[t], v[t])
        got.append(o)
    assert np.abs(np.stack(got) - want).max() < 1e-10
    assert np.abs(S - (c[-1] * S0 + (k * (c[-1] / c)[:, None]).T @ u)).max() < 1e-10


def test_delta_write_replaces_what_the_memory_holds_under_the_key():
    """Step size 1 and no decay: after writing (k, v) the memory answers k with v exactly, and an orthogonal key as before."""
    rng = np.random.default_rng(4)
    S = rng.standard_normal((3, 2))
    k, other, v = np.array([1.0, 0.0, 0.0]), np.array([0.0, 0.6, 0.8]), np.array([5.0, -2.0])
    before = S.T @ other
    S, o = O.delta_update(S, 1.0, 1.0, k, k, v)
    assert np.allclose(o, v) and np.allclose(S.T @ other, before)


def test_delta_gates():
    P = dict(b=np.array([[0.0], [800.0]]), a=np.array([[0.0], [-900.0]]), A_log=np.array([np.log(2.0), 0.0]), dt_bias=np.array([0.0, 0.0]))
    beta, g = O.delta_gates(P, np.array([1.0]))
    assert np.allclose(beta, [0.5, 1.0]) and np.allclose(g, [0.25, 1.0])       # exp(-2 ln 2), exp(-0)


def test_routing_inside_the_best_groups():
    r = dict(experts=6, top=2, groups=dict(count=3, keep=1), scale=1.5)
    s = np.array([0.9, 0.1, 0.6, 0.55, 0.5, 0.5])
    pick, w = O.route(s, np.zeros(6), r)
    assert list(pick) == [2, 3]                  # the pair's sum decides, not the best single expert
    assert np.allclose(w, 1.5 * s[[2, 3]] / 1.15)
    # the correction moves the choice and not the weight; scores below zero still beat closed groups
    c = np.array([-5.0, -5.0, -9.0, -9.0, -9.0, -9.0])
    pick, w = O.route(s, c, r)
    assert list(pick) == [0, 1] and np.allclose(w, 1.5 * s[[0, 1]] / 1.0)
    pick, w = O.route(s, np.zeros(6), dict(experts=6, top=3, groups=dict(count=6, keep=3), scale=1.0))      # groups of one
    assert list(pick) == [0, 2, 3]


def test_feed_forward_adds_the_shared_expert():
    cfg = make_config([delta(mlp=moe(experts=2, top=2, count=1, keep=1, scale=0.7))], width=10)
    P, mlp = params(cfg, 5, part="mlp."), cfg["layers"][0]["mlp"]
    h = np.random.default_rng(6).standard_normal(10)
    s = 1.0 / (1.0 + np.exp(-P["router"] @ h))

    def expert(n):
        z = P[n + ".gate"] @ h
        return P[n + ".down"] @ (z / (1.0 + np.exp(-z)) * (P[n + ".up"] @ h))

    want = 0.7 * (s[0] * expert("e0") + s[1] * expert("e1")) / s.sum()
    assert np.abs(O.experts_ff(P, dict(mlp, shared=None), h) - want).max() < 1e-10
    assert np.abs(O.experts_ff(P, mlp, h) - want - expert("shared")).max() < 1e-10


def test_sublayers_read_the_residual_itself_and_only_their_output_is_normed():
    cfg = make_config([attention(heads=1, kv_heads=1, window=1, mlp=None)], width=10)
    W = random_weights(cfg, seed=7)
    o = oracle_for(cfg, W)
    lg, lay = o.forward([5], return_layers=True)
    n = lambda v, w: v / np.sqrt((v * v).mean() + 1e-5) * (1.0 + w.astype(np.float64))
    x = n(W["embed"][5].astype(np.float64), W["embed.norm"])
    k = W["l0.mix.k"].astype(np.float64) @ x
    at = O.WindowAttention(O.sub(o.W, "l0.mix."), cfg["layers"][0]["mixer"], 1e-5)
    q, kn, v = at.project(x, 0)
    share = 1.0 / (1.0 + np.exp(o.W["l0.mix.sink"][0] - (q @ kn.T).item() * cfg["layers"][0]["mixer"]["scale"]))
    x = x + n(W["l0.mix.o"].astype(np.float64) @ (share * k), W["l0.norm1"])
    assert np.abs(lay[0, 0] - x).max() < 1e-10
    assert np.abs(lg[0] - W["head"].astype(np.float64) @ n(x, W["final.norm"])).max() < 1e-9


def test_a_planted_pair_decides_inside_the_window_only():
    cfg = make_config([attention(heads=2, kv_heads=1, dim=12, window=20, scale=3.0, mlp=None)], width=48, vocab=40)
    W = plant_pair(cfg, random_weights(cfg, seed=31, sink=(3.0, 0.2)), 7, 11)
    o = oracle_for(cfg, W)
    rng = np.random.default_rng(1)
    t = rng.integers(12, 40, size=40).tolist()
    t[39] = 7
    for back, visible in ((1, True), (19, True), (20, False), (30, False)):
        a = list(t)
        a[39 - back] = 11
        assert (rel_err(o.forward(a)[39:], o.forward(t)[39:])[0] > 0.3) == visible, back


@pytest.mark.parametrize("edit,what", [
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "kv_heads"),
    (lambda c: c["layers"][0]["mixer"].update(vdim=5), "vdim"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "mask"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=3), "rot"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=8), "rot"),
    (lambda c: c["layers"][0].update(type="retention"), "retention"),
    (lambda c: c["layers"][1]["mixer"].update(dim=1025), "dim"),
    (lambda c: c["layers"][1]["mixer"].update(conv=0), "conv"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=5), "router"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=4), "router"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=4), "router"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "mlp.kind"),
    (lambda c: c.pop("width"), "width"),
])
def test_a_config_that_makes_no_sense_is_refused_before_any_device_work(tmp_path, edit, what):
    from kubeai_b200 import B200Error
    from kubeai_b200.engine import Engine, default_config
    cfg = json.loads(json.dumps(make_config([attention(), delta()])))
    W = random_weights(cfg)
    edit(cfg)
    with pytest.raises(B200Error, match=what):
        Engine(default_config(manual_step=1), write_model_dir(tmp_path / "m", cfg, W), dtype="float32")
