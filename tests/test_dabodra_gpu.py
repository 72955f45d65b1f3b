"""Dabodra through the engine against the plain oracle (oracle/dabodra_oracle.py): each mechanism alone, prefill against
token-by-token decoding, portions down to two tokens, unequal batches, pages and slots used again, keys just inside and
just outside the window and far back found by a planted query/key pair, the sink, far tokens in the delta rule's state, the
carried inputs of its convolutions across cuts, routing whose choice hangs on one rule at a time, other sizes (also the
degenerate ones), long decoding, and greedy generation through the engine's own submit / scheduler / sampling path.
Configurations and weights are made here; nothing is read from disk but what the test wrote."""
import numpy as np
import pytest

from dabodra_util import (attention, bf16_round, delta, feed_portions, feed_whole, make_config, moe, open_engine, oracle_for, plant_pair,
                          random_weights, rel_err, write_model_dir)

pytestmark = pytest.mark.gpu

F32_TOL = 2e-5     # fp32 engine vs float64 oracle, relative RMS over the vocabulary


def close32(got, want, scale=1.0):
    r = rel_err(got, want)
    assert np.median(r) < F32_TOL * scale, np.median(r)
    assert r.max() < 15 * F32_TOL * scale, (int(np.argmax(r)), r.max())


def close16(got, want, most=0.95):
    """bf16 serving precision on these tiny widths: a percent or two per row.  The norm on every sublayer's output blows a
    nearly cancelling output up to full size with its rounding, and an expert choice that hangs on the last bits of the
    router's input may fall the other way, so a few rows may move further."""
    r = rel_err(got, want)
    assert np.median(r) < 0.03, np.median(r)
    assert np.quantile(r, most) < 0.15, np.quantile(r, most)


def toks(n, vocab, seed=0):
    return np.random.default_rng(seed).integers(0, vocab, size=n).tolist()


def build(tmp_path, layers, seed=0, wkw=None, edit=None, **kw):
    cfg = make_config(layers, **kw)
    W = random_weights(cfg, seed=seed, **(wkw or {}))
    if edit:
        edit(W)
        W = {k: bf16_round(v) for k, v in W.items()}
    return cfg, W, write_model_dir(tmp_path / "m", cfg, W)


# every kind of layer, with and without a feed-forward, unequal sizes and windows in neighbouring layers
MIX = [attention(), delta(mlp=None), attention(heads=6, kv_heads=1, dim=5, window=33, rot_dims=2, base=3000.0, mlp=None), delta(heads=3, kv_heads=3, dim=4, vdim=9, conv=4),
       attention(heads=3, kv_heads=3, dim=8, window=16, rot_dims=8, scale=0.5, mlp=moe(experts=4, top=1, count=1, keep=1, shared=0)),
       delta(heads=2, kv_heads=1, dim=11, vdim=3, conv=2, mlp=moe(experts=8, top=4, count=2, keep=1, ff=5, shared=9, scale=2.5))]


@pytest.fixture(scope="module")
def mix(tmp_path_factory):
    cfg, W, d = build(tmp_path_factory.mktemp("mix"), MIX)
    return cfg, W, d, oracle_for(cfg, W)


# ---------------------------------------------------------------- each mechanism alone
def fill(**values):
    def edit(W):
        for n, v in values.items():
            W["l0." + n.replace("__", ".")][...] = v
    return edit


@pytest.mark.parametrize("name,layers,kw,edit", [
    ("attention_only", [attention(mlp=None)], {}, None),
    ("attention_one_head_one_dimension", [attention(heads=1, kv_heads=1, dim=1, rot_dims=0, mlp=None)], {}, None),
    ("attention_a_key_head_per_head", [attention(heads=5, kv_heads=5, mlp=None)], {}, None),
    ("attention_one_key_head", [attention(heads=7, kv_heads=1, mlp=None)], {}, None),
    ("attention_three_heads_per_key_head", [attention(heads=6, kv_heads=2, dim=10, mlp=None)], {}, None),
    ("attention_unrotated", [attention(rot_dims=0, mlp=None)], {}, None),
    ("attention_all_dimensions_rotated", [attention(dim=6, rot_dims=6, base=7.0, mlp=None)], {}, None),
    ("attention_one_rotated_pair", [attention(dim=9, rot_dims=2, mlp=None)], {}, None),
    ("attention_window_of_one", [attention(heads=2, window=1, mlp=None)], {}, None),
    ("attention_window_of_two", [attention(window=2, mlp=None)], {}, None),
    ("attention_window_of_a_page", [attention(window=16, mlp=None)], {}, None),
    ("attention_window_past_the_end", [attention(window=1000, mlp=None)], {}, None),
    ("attention_unlike_windows", [attention(window=3, mlp=None), attention(window=20, mlp=None)], {}, None),
    ("attention_odd_scale", [attention(scale=1.7, mlp=None)], {}, None),
    ("attention_wide_head", [attention(heads=2, kv_heads=1, dim=200, rot_dims=64, mlp=None)], {}, None),
    ("attention_many_heads", [attention(heads=38, kv_heads=19, dim=4, rot_dims=2, mlp=None)], {}, None),
    ("attention_unlike_norm_weights", [attention(mlp=None)], {}, lambda W: (W["l0.mix.q.norm"].__setitem__(slice(0, 6), 3.0), W["l0.mix.k.norm"].__setitem__(slice(6, 12), -0.5))),
    ("delta_only", [delta(mlp=None)], {}, None),
    ("delta_one_of_each", [delta(heads=1, kv_heads=1, dim=1, vdim=2, conv=1, mlp=None)], {}, None),
    ("delta_a_key_head_per_head", [delta(heads=3, kv_heads=3, mlp=None)], {}, None),
    ("delta_one_key_head", [delta(heads=5, kv_heads=1, mlp=None)], {}, None),
    ("delta_one_tap", [delta(conv=1, mlp=None)], {}, None),
    ("delta_six_taps", [delta(conv=6, mlp=None)], {}, None),
    ("delta_many_rows", [delta(heads=2, kv_heads=1, dim=70, vdim=9, mlp=None)], {}, None),
    ("delta_more_rows_than_a_warp_holds_pieces", [delta(heads=2, kv_heads=2, dim=300, vdim=5, mlp=None)], {}, None),
    ("delta_wide_value", [delta(heads=2, kv_heads=1, dim=4, vdim=150, mlp=None)], {}, None),
    ("delta_no_decay", [delta(mlp=None)], {}, fill(mix__A_log=-60.0)),
    ("delta_full_decay", [delta(mlp=None)], {}, fill(mix__A_log=4.0, mix__dt_bias=9.0)),
    ("delta_large_step_sizes", [delta(mlp=None)], {}, lambda W: W["l0.mix.b"].__imul__(40.0)),
    ("delta_unlike_heads", [delta(heads=2, kv_heads=1, mlp=None)], {}, lambda W: (W["l0.mix.A_log"].__setitem__(slice(None), [-6.0, 2.0]), W["l0.mix.dt_bias"].__setitem__(slice(None), [1.0, -3.0]))),
    ("experts", [delta()], {}, None),
    ("experts_all_chosen", [delta(mlp=moe(experts=4, top=4, count=2, keep=2))], {}, None),
    ("experts_one", [attention(mlp=moe(experts=1, top=1, count=1, keep=1, ff=3, shared=1))], {}, None),
    ("experts_one_group", [attention(mlp=moe(experts=7, top=3, count=1, keep=1))], {}, None),
    ("experts_groups_of_one", [delta(mlp=moe(experts=6, top=2, count=6, keep=3))], {}, None),
    ("experts_groups_of_two", [delta(mlp=moe(experts=8, top=3, count=4, keep=2))], {}, None),
    ("experts_many_groups", [delta(mlp=moe(experts=48, top=5, count=16, keep=4, ff=3))], {}, None),
    ("experts_without_a_shared_one", [delta(mlp=moe(shared=0))], {}, None),
    ("experts_with_corrections_far_below_zero", [delta(mlp=moe(experts=6, top=4, count=3, keep=2))], {}, lambda W: W["l0.mlp.correction"].__isub__(5.0)),
    ("experts_ruled_by_the_correction", [delta(mlp=moe(experts=6, top=2, count=3, keep=1))], {}, lambda W: W["l0.mlp.correction"].__setitem__(slice(None), [1.5, 0, 0, -2, 1, 1])),
    ("experts_with_tiny_scores", [delta(mlp=moe(top=3))], {}, lambda W: W["l0.mlp.router"].__imul__(20.0)),
    ("no_feed_forward_at_all", [attention(mlp=None), delta(mlp=None)], {}, None),
    ("odd_width", [attention(), delta()], dict(width=21, vocab=33), None),
    ("large_eps_in_every_norm", [attention(), delta()], dict(eps=0.05), None),
])
def test_each_mechanism_matches_the_oracle(tmp_path, name, layers, kw, edit):
    cfg, W, d = build(tmp_path, layers, seed=3, edit=edit, **kw)
    o = oracle_for(cfg, W)
    t = toks(37, cfg["vocab"], 1)
    want, layers_want = o.forward(t, return_layers=True)
    with open_engine(d) as e:
        e.debug_residuals(True)
        got = feed_whole(e, t)
        res = e.read_residuals().reshape(layers_want.shape)
        e.debug_residuals(False)
        parts = feed_portions(e, t, [11, 2, 1])
    assert np.abs(res - layers_want).max() < 1e-4 * max(1.0, np.abs(layers_want).max()), name
    close32(got, want)
    close32(parts, want)


def test_sizes_the_config_leaves_to_the_tensors(tmp_path):
    """Taps and hidden sizes may stand in the checkpoint alone; what a mixer leaves out has its plain value."""
    import json
    layers = [delta(conv=4, mlp=moe(ff=11, shared=5)), attention(heads=3, kv_heads=3, dim=4, window=10 ** 6, scale=0.5, mlp=moe(count=1, keep=1, scale=1.0))]
    cfg, W, d = build(tmp_path, layers, seed=4)
    short = json.loads(json.dumps(cfg))
    del short["layers"][0]["mixer"]["conv"], short["layers"][0]["mlp"]["expert"], short["layers"][0]["mlp"]["shared"]["ff"]
    mx, ro = short["layers"][1]["mixer"], short["layers"][1]["mlp"]["router"]
    del mx["kv_heads"], mx["vdim"], mx["mask"], mx["scale"], ro["groups"], ro["scale"]
    t = toks(20, cfg["vocab"], 1)
    with open_engine(write_model_dir(tmp_path / "s", short, W)) as e:
        close32(feed_whole(e, t), oracle_for(cfg, W).forward(t))


def test_bfloat16_serving_precision_stays_near_the_oracle(mix):
    cfg, W, d, o = mix
    t = toks(70, cfg["vocab"], 2)
    want = o.forward(t)
    with open_engine(d, dtype="bfloat16") as e:
        close16(feed_whole(e, t), want, 0.8)
        close16(feed_portions(e, t, [40, 1]), want, 0.8)


MEDIUM = [attention(heads=6, kv_heads=2, dim=32, window=40, rot_dims=16, scale=0.15, mlp=moe(experts=4, top=2, count=2, keep=1, ff=104, shared=64)),
          delta(heads=4, kv_heads=2, dim=32, vdim=24, conv=4, mlp=moe(experts=6, top=3, count=3, keep=2, ff=40, shared=256)),
          attention(heads=4, kv_heads=4, dim=16, window=100, rot_dims=16, scale=0.2, mlp=None), delta(heads=2, kv_heads=2, dim=48, vdim=40, conv=3, mlp=None)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seqs", [1, 5, 12, 17])
def test_decode_batches_of_every_width(tmp_path, dtype, seqs):
    """Steps of one token per sequence at batch sizes on both sides of the few-row product kernels' limits and of the limit
    of the per-pair expert path; fp32 results per row must not depend on the batch."""
    cfg, W, d = build(tmp_path, MEDIUM, seed=19, width=88, vocab=100)
    o = oracle_for(cfg, W)
    ts = [toks(9, 100, 20 + i) for i in range(seqs)]
    with open_engine(d, dtype=dtype, max_tokens=64, max_seqs=seqs, budget=256) as e:
        rids = [e.feed_open() for _ in ts]
        e.feed_step([(r, t[:4], []) for r, t in zip(rids, ts)])
        got = [e.feed_step([(r, [t[k]], [0]) for r, t in zip(rids, ts)]) for k in range(4, 9)]
        for r in rids:
            e.feed_close(r)
    want = np.stack([o.forward(t)[4:] for t in ts], axis=1)
    (close32 if dtype == "float32" else lambda a, b: close16(a, b, 0.85))(np.concatenate(got), want.reshape(-1, 100))


def test_bfloat16_widths_the_tensor_core_projection_cannot_take(tmp_path):
    """A width and inner sizes that are no multiple of 8 run on the general linear kernels."""
    cfg, W, d = build(tmp_path, [attention(heads=3, kv_heads=1, dim=5), delta(heads=3, kv_heads=3, dim=5, vdim=3, mlp=None)], width=20, vocab=33)
    t = toks(40, 33, 4)
    want = oracle_for(cfg, W).forward(t)
    with open_engine(d, dtype="bfloat16") as e:
        close16(feed_whole(e, t), want, 0.8)
        close16(feed_portions(e, t, [20, 3, 1]), want, 0.8)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_medium_sizes_on_every_projection_and_expert_path(tmp_path, dtype):
    """Steps of 300 tokens (a GEMM per expert in bf16), tens of tokens (grouped 64-row tiles) and single ones (a pass per
    chosen pair)."""
    cfg, W, d = build(tmp_path, MEDIUM, seed=17, width=72, vocab=90)
    t = toks(460, 90, 18)
    want = oracle_for(cfg, W).forward(t)
    with open_engine(d, dtype=dtype) as e:
        whole = feed_whole(e, t)
        parts = feed_portions(e, t, [300, 9, 33, 16, 1])
    check = close32 if dtype == "float32" else (lambda a, b: close16(a, b, 0.85))
    check(whole, want)
    check(parts, want)


def test_whole_tile_products_of_large_steps_equal_the_stream_k_ones(tmp_path, monkeypatch):
    """Steps of more than 256 tokens take whole-tile products, the shared expert with its gated unit in the epilogue; the last
    token tiles and the last weight tiles are partial.  All rows are those of the stream-K form with a pass of its own."""
    layers = [attention(heads=16, kv_heads=4, dim=64, window=300, rot_dims=32, scale=0.125, mlp=moe(experts=2, top=1, count=1, keep=1, ff=64, shared=1984)),
              delta(heads=8, kv_heads=4, dim=96, vdim=120, conv=4, mlp=None)]
    cfg, W, d = build(tmp_path, layers, seed=81, width=2048, vocab=64)
    T = 4700
    t = toks(T, 64, 82)
    rows = sorted(set(range(24)) | set(range(100, T, 97)) | {255, 256, 511, 512, 4095, 4096, 4607, 4608, T - 1})
    out = {}
    for knob in ("1", "0"):
        monkeypatch.setenv("B200_DB_WHOLE", knob)
        with open_engine(d, dtype="bfloat16", max_tokens=4704, max_seqs=1) as e:
            out[knob] = feed_whole(e, t, rows)
    close16(out["1"][:24], oracle_for(cfg, W).forward(t[:24]))
    r = rel_err(out["1"], out["0"].astype(np.float64))
    assert np.median(r) < 0.01 and np.quantile(r, 0.95) < 0.05, (np.median(r), r.max())


@pytest.mark.parametrize("experts,top,ff,width,T", [(4, 2, 64, 72, 700), (16, 2, 192, 64, 300), (3, 1, 40, 136, 1000), (40, 8, 64, 64, 61), (8, 3, 8, 256, 33), (2, 2, 640, 264, 513), (6, 1, 128, 8, 90)])
def test_grouped_expert_products_equal_the_plain_ones(tmp_path, monkeypatch, experts, top, ff, width, T):
    """Experts of no, few and hundreds of rows (several row tiles), hidden sizes with the gated unit in the epilogue (multiples of
    64) and without, partial weight tiles and k-blocks: every row is the one that the plain grouped kernels give."""
    cfg, W, d = build(tmp_path, [delta(heads=2, kv_heads=1, dim=8, vdim=8, conv=1, mlp=moe(experts=experts, top=top, count=1, keep=1, ff=ff, shared=16))], seed=51, width=width, vocab=60,
                      edit=lambda W: W["l0.mlp.correction"].__setitem__(slice(None), np.where(np.arange(experts) == experts - 1, -3.0, np.where(np.arange(experts) == 0, 0.4, 0.0))))
    t = toks(T, 60, 52)
    out = {}
    for knob in ("1", "0"):
        monkeypatch.setenv("B200_DB_GROUPED", knob)
        with open_engine(d, dtype="bfloat16", max_tokens=1024, max_seqs=1) as e:
            out[knob] = feed_whole(e, t)
    close16(out["1"][:40], oracle_for(cfg, W).forward(t[:40]), 0.8)
    r = rel_err(out["1"], out["0"].astype(np.float64))
    assert np.median(r) < 0.01 and r.max() < 0.06, (np.median(r), r.max())


@pytest.mark.parametrize("heads,kv_heads,dim,window", [(4, 2, 16, 70), (6, 1, 32, 17), (8, 8, 64, 64), (16, 1, 128, 100), (5, 5, 48, 1), (64, 1, 16, 128), (2, 1, 112, 333)])
def test_bfloat16_tensor_core_attention_equals_the_general_kernel(tmp_path, monkeypatch, heads, kv_heads, dim, window):
    """Head sizes that fit the mma fragments, with a sink per head: the 64-row kernel against the general one on the same
    bf16 cache, with windows inside, across and beyond a key tile, and portions cut anywhere."""
    cfg, W, d = build(tmp_path, [attention(heads=heads, kv_heads=kv_heads, dim=dim, window=window, rot_dims=dim // 2, scale=0.5 * dim ** -0.5, mlp=None)],
                      seed=21, width=64, vocab=60, wkw=dict(sink=(1.0, 1.5)))
    t = toks(230, 60, 22)
    want = oracle_for(cfg, W).forward(t)
    out = {}
    for knob in ("1", "0"):
        monkeypatch.setenv("B200_WATTN_MMA", knob)
        with open_engine(d, dtype="bfloat16") as e:
            out[knob] = (feed_whole(e, t), feed_portions(e, t, [67, 2, 90, 1]))
    for a, b in zip(out["1"], out["0"]):
        close16(a, want)
        r = rel_err(a, b.astype(np.float64))
        assert np.median(r) < 0.02 and np.quantile(r, 0.98) < 0.1, (np.median(r), r.max())


@pytest.mark.parametrize("heads,kv_heads,dim,vdim", [(4, 2, 16, 16), (3, 3, 128, 64), (6, 2, 48, 24), (2, 1, 64, 136), (8, 1, 112, 8), (5, 5, 32, 72), (2, 2, 80, 128), (1, 1, 128, 200)])
def test_chunked_tensor_core_scan_equals_the_token_by_token_scan(tmp_path, monkeypatch, heads, kv_heads, dim, vdim):
    """Sizes that the chunked form takes (whole and partial blocks of key rows and value columns, several chunks of 64,
    portions that end inside a chunk or a 16-token block): it keeps fp32 precision, so only the rounding of the layer's
    bf16 output can differ from the sequential scan."""
    cfg, W, d = build(tmp_path, [delta(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=4, mlp=None)], seed=5, width=64, vocab=60, wkw=dict(a_log=(-5.0, 0.0)))
    t = toks(333, 60, 6)
    want = oracle_for(cfg, W).forward(t)
    out = {}
    for knob in ("1", "0"):          # from one token per portion; never
        monkeypatch.setenv("B200_DELTA_CHUNK", knob)
        with open_engine(d, dtype="bfloat16") as e:
            out[knob] = (feed_whole(e, t), feed_portions(e, t, [100, 64, 1, 17, 2, 90, 1]))
    for a, b in zip(out["1"], out["0"]):
        close16(a, want)
        r = rel_err(a, b.astype(np.float64))
        assert np.median(r) < 1e-3 and r.max() < 0.01, (np.median(r), r.max())


@pytest.mark.parametrize("a_log,dt_bias,b_gain", [(4.0, 9.0, 1.0), (-9.0, -2.0, 1.0), (-9.0, -60.0, 60.0), (2.0, 3.0, 60.0)])
def test_chunked_scan_at_extreme_gates(tmp_path, monkeypatch, a_log, dt_bias, b_gain):
    """Decays that leave nothing of a state after one token (no factor may overflow), decays next to one, step sizes of all
    but zero and all but one, and only a few different keys, so that most writes overwrite an earlier one."""
    cfg, W, d = build(tmp_path, [delta(heads=4, kv_heads=2, dim=32, vdim=32, conv=1, mlp=None)], seed=7, width=48, vocab=6,
                      edit=lambda W: (W["l0.mix.A_log"].fill(a_log), W["l0.mix.dt_bias"].fill(dt_bias), W["l0.mix.b"].__imul__(b_gain)))
    t = toks(200, 6, 8)
    want = oracle_for(cfg, W).forward(t)
    with open_engine(d, dtype="bfloat16") as e:
        got = feed_whole(e, t)
    monkeypatch.setenv("B200_DELTA_CHUNK", "0")
    with open_engine(d, dtype="bfloat16") as e:
        one = feed_whole(e, t)
    assert np.isfinite(got).all()
    close16(got, want)
    assert rel_err(got, one.astype(np.float64)).max() < 0.02


def test_chunked_scan_behind_strong_decays_keeps_the_weak_ones(tmp_path, monkeypatch):
    """One token forgets everything (its log decay is in the thousands), the others nearly nothing: the decays between later
    tokens of the same chunk are differences of large sums and must keep their low bits."""
    def edit(W):
        a = np.zeros_like(W["l0.mix.a"])
        x = W["embed"][0].astype(np.float64)
        x = x / np.sqrt((x * x).mean() + 1e-5) * (1.0 + W["embed.norm"])
        a[:] = 3000.0 * x / (x @ x)
        W["l0.mix.a"] = bf16_round(a)
        W["l0.mix.dt_bias"].fill(-4.0)
        W["l0.mix.A_log"].fill(0.0)
    cfg, W, d = build(tmp_path, [delta(heads=2, kv_heads=1, dim=16, vdim=16, conv=1, mlp=None)], seed=9, width=48, vocab=40, edit=edit)
    H = np.stack([oracle_for(cfg, W).norm("embed.norm", W["embed"][v].astype(np.float64)) for v in range(40)]) @ W["l0.mix.a"][0].astype(np.float64)
    calm = [v for v in range(1, 40) if H[v] < 0]
    t = [calm[i] for i in np.random.default_rng(10).integers(0, len(calm), size=100)]
    t[3] = t[37] = t[70] = 0
    want = oracle_for(cfg, W).forward(t)
    out = []
    for knob in ("8", "0"):
        monkeypatch.setenv("B200_DELTA_CHUNK", knob)
        with open_engine(d, dtype="bfloat16") as e:
            out.append(feed_whole(e, t))
    close16(out[0], want)
    assert rel_err(out[0], out[1].astype(np.float64)).max() < 0.01


# ---------------------------------------------------------------- cutting a sequence
def test_prefill_equals_token_by_token_decoding(mix):
    cfg, W, d, o = mix
    t = toks(45, cfg["vocab"], 3)
    with open_engine(d) as e:
        whole = feed_whole(e, t)
        single = feed_portions(e, t, [1])
    close32(whole, o.forward(t))
    assert np.abs(whole - single).max() < 2e-4 * np.abs(whole).max()


@pytest.mark.parametrize("sizes", [[2], [3, 2], [16, 1], [17, 5, 2], [5, 16, 16, 2, 1], [1, 1, 2, 1, 3]])
def test_portions_of_any_size_give_the_same_logits(mix, sizes):
    cfg, W, d, o = mix
    t = toks(61, cfg["vocab"], 5)
    with open_engine(d) as e:
        close32(feed_portions(e, t, sizes), o.forward(t))


@pytest.mark.parametrize("taps", [2, 4, 7])
def test_carried_convolution_inputs_survive_portions_shorter_than_the_taps(tmp_path, taps):
    """Portions of one and two tokens under a convolution of up to seven taps: the slot's carried inputs are shifted, not
    replaced, and a later portion still reads inputs of three steps ago."""
    cfg, W, d = build(tmp_path, [delta(conv=taps, mlp=None), delta(heads=2, kv_heads=2, conv=taps, vdim=12, mlp=None)], seed=6)
    t = toks(33, cfg["vocab"], 7)
    want = oracle_for(cfg, W).forward(t)
    with open_engine(d) as e:
        close32(feed_portions(e, t, [1, 2, 1, 1, 2, 5, 1, 2, 2, 1]), want)
        close32(feed_portions(e, t, [taps - 1, taps, 1, taps + 1, 2]), want)


def test_long_decoding_stays_on_the_oracle(tmp_path):
    """A window that passes over decoded tokens many times, pages behind it going back to the pool, beside a long-lived state."""
    cfg, W, d = build(tmp_path, [attention(window=21), delta(mlp=None), attention(window=5, mlp=None)], seed=8, wkw=dict(a_log=(-6.0, -3.0)))
    t = toks(300, cfg["vocab"], 7)
    want = oracle_for(cfg, W).forward(t)
    with open_engine(d) as e:
        got = feed_portions(e, t, [20, 1])
    close32(got, want, 5)


# ---------------------------------------------------------------- batches, pages, slots
def run_plan(e, seqs, plan):
    """Feed the sequences side by side: plan[step][i] tokens of sequence i per step (0: it sits the step out; past the plan's
    end every unfinished sequence brings one token).  Returns every sequence's logits."""
    rids = [e.feed_open() for _ in seqs]
    at, got, step = [0] * len(seqs), [[] for _ in seqs], 0
    while any(at[i] < len(seqs[i]) for i in range(len(seqs))):
        entries, idx = [], []
        for i in range(len(seqs)):
            n = min(plan[min(step, len(plan) - 1)][i] or (1 if step >= len(plan) else 0), len(seqs[i]) - at[i])
            if n > 0:
                entries.append((rids[i], seqs[i][at[i]:at[i] + n], list(range(n))))
                idx.append((i, n))
        out = e.feed_step(entries)
        r = 0
        for i, n in idx:
            got[i].append(out[r:r + n])
            at[i] += n
            r += n
        step += 1
    for r in rids:
        e.feed_close(r)
    return [np.concatenate(g) for g in got]


def test_unequal_requests_in_one_batch_equal_each_alone(mix):
    cfg, W, d, o = mix
    seqs = [toks(n, cfg["vocab"], 10 + i) for i, n in enumerate((50, 23, 9, 77))]
    plan = [(7, 1, 9, 30), (20, 1, 0, 2), (1, 3, 0, 17), (22, 1, 0, 1), (0, 17, 0, 27)]
    with open_engine(d, max_tokens=128) as e:
        got = run_plan(e, seqs, plan)
    for i in range(4):
        close32(got[i], o.forward(seqs[i]))


def test_bfloat16_mixed_batches_on_the_tensor_core_kernels_equal_each_request_alone(tmp_path):
    layers = [attention(heads=4, kv_heads=2, dim=16, window=37, rot_dims=8, mlp=None), delta(heads=4, kv_heads=2, dim=16, vdim=16, conv=4, mlp=None),
              attention(heads=8, kv_heads=1, dim=32, window=64, rot_dims=32, mlp=None), delta(heads=2, kv_heads=2, dim=64, vdim=32, mlp=None)]
    cfg, W, d = build(tmp_path, layers, seed=71, width=64)
    o = oracle_for(cfg, W)
    seqs = [toks(n, cfg["vocab"], 72 + i) for i, n in enumerate((150, 61, 9, 120))]
    plan = [(70, 1, 9, 33), (37, 1, 0, 2), (1, 40, 0, 64), (42, 1, 0, 1), (0, 18, 0, 20)]
    with open_engine(d, dtype="bfloat16", max_tokens=160) as e:
        got = run_plan(e, seqs, plan)
        alone = [feed_whole(e, t) for t in seqs]
    for i in range(4):
        close16(got[i], o.forward(seqs[i]))
        r = rel_err(got[i], alone[i].astype(np.float64))
        assert np.median(r) < 0.02 and np.quantile(r, 0.95) < 0.1


def feed_portions_on(e, r, tokens, sizes):
    outs, at, i = [], 0, 0
    while at < len(tokens):
        n = min(sizes[min(i, len(sizes) - 1)], len(tokens) - at)
        outs.append(e.feed_step([(r, tokens[at:at + n], list(range(n)))]))
        at += n
        i += 1
    e.feed_close(r)
    return np.concatenate(outs)


# windows past every sequence below, so that no page goes back early
WIDE = [attention(window=64), delta(mlp=None), attention(heads=6, kv_heads=1, dim=5, window=200, rot_dims=2, mlp=None), delta(heads=3, kv_heads=3, dim=4, vdim=9, conv=4)]


@pytest.fixture(scope="module")
def wide(tmp_path_factory):
    cfg, W, d = build(tmp_path_factory.mktemp("wide"), WIDE, seed=2)
    return cfg, W, d, oracle_for(cfg, W)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_pages_and_slots_are_used_again(wide, dtype):
    """A pool of exactly two sequences' pages and two slots: later requests run in what earlier ones gave back, and start
    from empty states and empty carried inputs whatever the slot held."""
    cfg, W, d, o = wide
    check = close32 if dtype == "float32" else (lambda a, b: close16(a, b, 0.8))
    seqs = [toks(n, cfg["vocab"], 20 + i) for i, n in enumerate((40, 33, 48, 17, 41))]
    with open_engine(d, dtype=dtype, max_tokens=48, max_seqs=2, blocks=6, budget=96) as e:
        a, b = e.feed_open(), e.feed_open()
        e.feed_step([(a, seqs[0], []), (b, seqs[1][:20], [])])
        e.feed_step([(b, seqs[1][20:], [])])
        e.feed_close(a)
        c = e.feed_open()                      # takes a's slot and pages while b is still live
        got_c = e.feed_step([(c, seqs[2][:30], list(range(30)))])
        e.feed_close(b)
        f = e.feed_open()
        out = e.feed_step([(c, seqs[2][30:], list(range(18))), (f, seqs[3], list(range(17)))])
        got_c = np.concatenate([got_c, out[:18]])
        got_f = out[18:]
        e.feed_close(c)
        e.feed_close(f)
        g = e.feed_open()
        got_g = feed_portions_on(e, g, seqs[4], [16, 1])
        assert e.stats().kv_blocks_free == 6
    check(got_c, o.forward(seqs[2]))
    check(got_f, o.forward(seqs[3]))
    check(got_g, o.forward(seqs[4]))


def test_a_step_over_the_pool_is_refused_and_leaves_the_engine_usable(wide):
    from kubeai_b200 import B200Error
    cfg, W, d, o = wide
    t = toks(40, cfg["vocab"], 30)
    with open_engine(d, max_tokens=48, max_seqs=2, blocks=3) as e:
        a, b = e.feed_open(), e.feed_open()
        e.feed_step([(a, t[:30], [])])
        with pytest.raises(B200Error):
            e.feed_step([(b, t[:30], [])])        # 2 + 2 pages do not fit 3
        got = e.feed_step([(a, t[30:], list(range(10)))])
        e.feed_close(a)
        e.feed_close(b)
    close32(got, o.forward(t)[30:])


def test_pages_behind_the_window_return_to_the_pool_while_the_sequence_runs(tmp_path):
    """Two sequences far longer than the pool could hold side by side, windows of different layers up to 20 tokens."""
    cfg, W, d = build(tmp_path, [attention(window=20), delta(mlp=None), attention(window=7, mlp=None)], seed=35)
    o = oracle_for(cfg, W)
    seqs = [toks(150, cfg["vocab"], 36), toks(140, cfg["vocab"], 37)]
    with open_engine(d, max_tokens=160, max_seqs=2, blocks=10, budget=64) as e:
        got = run_plan(e, seqs, [(16, 10), (10, 16), (1, 1), (5, 2)] + [(3, 4)] * 30)
        assert e.stats().kv_blocks_free == 10
    for k in range(2):
        close32(got[k], o.forward(seqs[k]), 2)


def test_a_model_without_attention_and_one_without_recurrence(tmp_path):
    for i, layers in enumerate(([delta(), delta(mlp=None)], [attention(), attention(window=30, mlp=None)])):
        cfg, W, d = build(tmp_path / str(i), layers, seed=33 + i)
        o = oracle_for(cfg, W)
        seqs = [toks(n, cfg["vocab"], 34 + k) for k, n in enumerate((30, 12))]
        with open_engine(d, max_tokens=64, max_seqs=2) as e:
            got = run_plan(e, seqs, [(9, 1), (1, 3), (20, 0)])
        for k in range(2):
            close32(got[k], o.forward(seqs[k]))


# ---------------------------------------------------------------- single keys made visible
QTOK, KTOK = 7, 11


def planted_model(tmp_path, window, dim=16):
    """One attention layer that copies from KTOK positions whenever a QTOK position sees one (planted pair, sharp softmax)."""
    cfg = make_config([attention(heads=2, kv_heads=1, dim=dim, window=window, rot_dims=4, scale=2.0, mlp=None)], width=48, vocab=40)
    W = plant_pair(cfg, random_weights(cfg, seed=31, sink=(3.0, 0.2)), QTOK, KTOK)
    return cfg, W, write_model_dir(tmp_path / "m", cfg, W), oracle_for(cfg, W)


def sequence_with(n, marks, seed):
    """Random filler without the two special tokens, marks[position] = token."""
    t = np.random.default_rng(seed).integers(12, 40, size=n).tolist()
    for p, x in marks.items():
        t[p] = x
    return t


@pytest.mark.parametrize("window", [2, 5, 15, 16, 17, 63, 64, 65, 100, 130])
def test_the_windows_edge_in_prompts_and_in_decoding(tmp_path, window):
    """The key window - 1 positions back decides the query's logits and the key `window` positions back does not, wherever
    the pair lies against pages and tiles, whole, cut between and around the two, and decoded."""
    cfg, W, d, o = planted_model(tmp_path, window)
    with open_engine(d) as e32, open_engine(d, dtype="bfloat16") as e16:
        for first in (0, 1, 15, 16, 47, 64):
            q_in, q_out = first + window - 1, first + window
            n = q_out + 3
            for q, visible in ((q_in, True), (q_out, False)):
                t = sequence_with(n, {first: KTOK, q: QTOK}, first)
                gone = list(t)
                gone[first] = 13
                want = o.forward(t)
                differs = rel_err(want[q:q + 1], o.forward(gone)[q:q + 1])[0]
                assert differs > 0.3 if visible else differs < 1e-12
                for got in (feed_whole(e32, t), feed_portions(e32, t, [first + 1, max(1, q - first - 1), 1]), feed_portions(e32, t, [max(1, q), 1]),
                            feed_portions(e32, t, [max(1, q - 1), 2, 1])):
                    close32(got, want, 2)
                for got in (feed_whole(e16, t), feed_portions(e16, t, [max(1, q), 1])):
                    assert rel_err(got, want)[q] < 0.2


@pytest.mark.parametrize("key,query", [(0, 15), (0, 16), (15, 16), (31, 400), (0, 447), (63, 64), (64, 128), (255, 440), (1, 2)])
def test_a_far_key_is_found_wherever_it_lies(tmp_path, key, query):
    cfg, W, d, o = planted_model(tmp_path, 500)
    n = query + 3
    t = sequence_with(n, {key: KTOK, query: QTOK}, 1)
    gone = list(t)
    gone[key] = 13
    want = o.forward(t)
    assert rel_err(want[query:query + 1], o.forward(gone)[query:query + 1])[0] > 0.3      # the key decides
    with open_engine(d) as e:
        close32(feed_whole(e, t), want, 2)
        close32(feed_portions(e, t, [key + 1, max(1, query - key - 1), 1]), want, 2)
        close32(feed_portions(e, t, [query, 1]), want, 2)
    with open_engine(d, dtype="bfloat16") as e:
        for got in (feed_whole(e, t), feed_portions(e, t, [query, 1])):
            r = rel_err(got, want)
            assert np.median(r) < 0.05 and r[query] < 0.2


@pytest.mark.parametrize("query", [15, 16, 31, 63, 64, 200])
def test_a_key_behind_the_query_is_not_seen(tmp_path, query):
    """The token after the query (in the same step, page or tile) would decide its logits if it were visible."""
    cfg, W, d, o = planted_model(tmp_path, 90)
    t = sequence_with(query + 6, {query: QTOK, query + 1: KTOK, query + 2: KTOK}, 2)
    plain = list(t)
    plain[query + 1], plain[query + 2] = 14, 15
    want = o.forward(t)
    with open_engine(d) as e:
        a, b = feed_whole(e, t), feed_whole(e, plain)
        assert np.abs(a[query] - b[query]).max() < 1e-4 * np.abs(a[query]).max()
        close32(a, want, 2)
        close32(feed_portions(e, t, [query + 1, 2, 1]), want, 2)
    with open_engine(d, dtype="bfloat16") as e:
        assert rel_err(feed_whole(e, t), want)[query] < 0.2


def test_a_far_key_survives_other_requests_in_the_batch(tmp_path):
    cfg, W, d, o = planted_model(tmp_path, 195)
    a = sequence_with(200, {3: KTOK, 197: QTOK}, 5)
    b = sequence_with(90, {60: KTOK, 88: QTOK}, 6)
    c = sequence_with(70, {69: QTOK}, 7)          # no key of its own: it must not find the others'
    with open_engine(d, max_tokens=208) as e:
        got = run_plan(e, [a, b, c], [(100, 30, 2), (33, 1, 30), (60, 55, 30), (3, 1, 5)])
    for g, t in zip(got, (a, b, c)):
        close32(g, o.forward(t), 2)


def test_the_sink_takes_its_share_of_the_softmax(tmp_path):
    """Sinks that empty one head and leave the other, in both orders, sinks that leave the plain softmax, and ones far out of
    range: the engine follows the oracle, and the outputs differ (the norm behind the mixer hides only a common factor)."""
    cfg = make_config([attention(heads=2, kv_heads=1, dim=16, window=30, rot_dims=8, mlp=None)])
    W = random_weights(cfg, seed=15)
    t = toks(90, cfg["vocab"], 16)
    outs = []
    for i, sink in enumerate(([6.0, -30.0], [-30.0, 6.0], [-30.0, -30.0], [3.0, 1.0], [90.0, -1e4])):
        Ws = dict(W)
        Ws["l0.mix.sink"] = bf16_round(np.array(sink, dtype=np.float32))
        d = write_model_dir(tmp_path / ("s%d" % i), cfg, Ws)
        want = oracle_for(cfg, Ws).forward(t)
        with open_engine(d) as e:
            close32(feed_whole(e, t), want)
            close32(feed_portions(e, t, [13, 70, 1]), want)
        with open_engine(d, dtype="bfloat16") as e:
            close16(feed_whole(e, t), want)
            close16(feed_portions(e, t, [13, 70, 1]), want)
        outs.append(want)
    assert min(rel_err(outs[i], outs[j]).max() for i, j in ((0, 1), (0, 2), (1, 2), (2, 3))) > 0.05


def test_distance_turns_the_rotated_scores(tmp_path):
    """With every dimension rotated and a sharp softmax, positions far into a sequence still see the right angles."""
    cfg, W, d = build(tmp_path, [attention(heads=2, kv_heads=2, dim=8, rot_dims=8, base=50000.0, scale=1.5, window=400, mlp=None)], seed=25)
    t = toks(420, cfg["vocab"], 26)
    want = oracle_for(cfg, W).forward(t)
    with open_engine(d) as e:
        close32(feed_whole(e, t), want, 2)
        close32(feed_portions(e, t, [333, 40, 1]), want, 2)


# ---------------------------------------------------------------- the delta rule's memory
def test_far_tokens_reach_through_the_state(tmp_path):
    """With decays next to one and small steps the state carries the first tokens across hundreds of positions: other first
    tokens change the last logits, and the engine follows the oracle whole, in portions and decoded."""
    cfg, W, d = build(tmp_path, [delta(heads=2, kv_heads=1, dim=16, vdim=16, mlp=None)], seed=41, edit=lambda W: (W["l0.mix.A_log"].fill(-9.0), W["l0.mix.b"].__imul__(4.0)))
    o = oracle_for(cfg, W)
    a = toks(300, cfg["vocab"], 42)
    b = [(x + 1) % cfg["vocab"] for x in a[:20]] + a[20:]
    wa, wb = o.forward(a), o.forward(b)
    assert rel_err(wa[-1:], wb[-1:])[0] > 1e-3
    with open_engine(d) as e:
        close32(feed_whole(e, a), wa, 3)
        close32(feed_portions(e, b, [150, 33, 1]), wb, 3)
    with open_engine(d, dtype="bfloat16") as e:
        close16(feed_whole(e, a), wa)


def test_a_second_write_under_the_same_key_replaces_the_first(tmp_path):
    """Steps of one half, no decay, one tap, one token again and again, queries equal to keys: the memory's answer approaches
    that token's value and stays there (an additive memory would grow without end)."""
    cfg, W, d = build(tmp_path, [delta(heads=2, kv_heads=2, dim=8, vdim=6, conv=1, mlp=None)], seed=43, vocab=12,
                      edit=lambda W: (W["l0.mix.A_log"].fill(-60.0), W["l0.mix.q"].__setitem__(slice(None), W["l0.mix.k"]), W["l0.mix.q.conv"].__setitem__(slice(None), W["l0.mix.k.conv"]),
                                      W["l0.mix.b"].fill(0.0)))
    o = oracle_for(cfg, W)
    t = [3, 3, 3, 3, 3, 3, 3, 3]
    want = o.forward(t)
    with open_engine(d) as e:
        close32(feed_whole(e, t), want)
        close32(feed_portions(e, t, [3, 1]), want)
    # step size 1/2 each time: the answers approach the value, o_n = (1 - 2^-n) v, and the norm behind them cancels the factor
    assert rel_err(want[1:], want[:1]).max() < 1e-3      # up to eps


def test_first_tokens_of_a_sequence(mix):
    cfg, W, d, o = mix
    with open_engine(d) as e:
        for n in (1, 2, 3):
            t = toks(n, cfg["vocab"], 50 + n)
            close32(feed_whole(e, t), o.forward(t))
        t = toks(6, cfg["vocab"], 54)
        close32(feed_portions(e, t, [1, 1, 2]), o.forward(t))


# ---------------------------------------------------------------- routing, one rule at a time
def test_routing_rules_decide_visibly(tmp_path):
    """The oracle with one rule changed gives other logits, the engine gives the oracle's: the two best members rank a group
    (not the best one), closed groups count as minus infinity (corrections below zero), the correction ranks and does not
    weigh, the weights are shares times the constant."""
    from oracle import dabodra_oracle as O
    cfg, W, d = build(tmp_path, [delta(mlp=moe(experts=9, top=3, count=3, keep=1, scale=2.2)), attention()], seed=61, edit=lambda W: W["l0.mlp.correction"].__isub__(1.5))
    t = toks(60, cfg["vocab"], 62)
    want = oracle_for(cfg, W).forward(t)
    with open_engine(d) as e:
        close32(feed_whole(e, t), want)
        close32(feed_portions(e, t, [30, 7, 1]), want)

    def other(s, correction, router, best_only=False, zero=False, weigh=False, raw=False):
        c = s + correction
        gr = router["groups"]
        parts = c.reshape(gr["count"], -1)
        rank = np.sort(parts, axis=1)[:, -1:].sum(axis=1) if best_only else np.sort(parts, axis=1)[:, -2:].sum(axis=1)
        open_ = np.repeat(np.isin(np.arange(gr["count"]), np.argsort(-rank, kind="stable")[:gr["keep"]]), parts.shape[1])
        pick = np.argsort(-np.where(open_, c, 0.0 if zero else -np.inf), kind="stable")[:router["top"]]
        w = c[pick] if weigh else s[pick]
        return pick, w if raw else w / (w.sum() + 1e-20) * router["scale"]

    plain = O.route
    for rule in ("best_only", "zero", "weigh", "raw"):
        O.route = lambda s, c, r: other(s, c, r, **{rule: True})
        try:
            assert rel_err(oracle_for(cfg, W).forward(t), want).max() > 0.05, rule
        finally:
            O.route = plain


# ---------------------------------------------------------------- random configurations
def random_layers(rng, n, size):
    layers = []
    for _ in range(n):
        G = int(rng.integers(1, 4))
        H = G * int(rng.integers(1, 4))
        count = int(rng.integers(1, 4))
        per, keep = int(rng.integers(1, 4)), int(rng.integers(1, count + 1))
        mlp = None if rng.random() < 0.3 else moe(experts=count * per, top=int(rng.integers(1, keep * per + 1)), count=count, keep=keep, ff=size(20),
                                                  shared=0 if rng.random() < 0.3 else size(20), scale=float(rng.uniform(0.5, 3.0)))
        D = size(14)
        if rng.random() < 0.5:
            layers.append(attention(heads=H, kv_heads=G, dim=D, window=int(rng.integers(1, 60)), rot_dims=2 * int(rng.integers(0, D // 2 + 1)),
                                    base=float(rng.choice([30.0, 1e4, 5e5])), scale=float(rng.uniform(0.3, 1.2)) * D ** -0.5, mlp=mlp))
        else:
            layers.append(delta(heads=H, kv_heads=G, dim=D, vdim=size(14), conv=int(rng.integers(1, 6)), mlp=mlp))
    return layers


@pytest.mark.parametrize("seed", range(10))
def test_random_configurations(tmp_path, seed):
    rng = np.random.default_rng(100 + seed)
    layers = random_layers(rng, int(rng.integers(1, 6)), lambda hi: int(rng.integers(2, hi)))
    cfg, W, d = build(tmp_path, layers, seed=200 + seed, width=int(rng.integers(6, 40)), vocab=int(rng.integers(5, 60)))
    t = toks(70, cfg["vocab"], seed)
    want = oracle_for(cfg, W).forward(t)
    with open_engine(d) as e:
        close32(feed_whole(e, t), want, 4)
        close32(feed_portions(e, t, [int(rng.integers(2, 30)), int(rng.integers(1, 9)), 1]), want, 4)


@pytest.mark.parametrize("seed", range(5))
def test_bfloat16_random_medium_configurations(tmp_path, seed):
    """Sizes that the tensor-core projections, attention and scan take (multiples of 16), in random layer orders: the bf16
    engine stays near the oracle whole and in portions, and the fp32 engine on all rows."""
    rng = np.random.default_rng(300 + seed)
    layers = random_layers(rng, int(rng.integers(2, 5)), lambda hi: 16 * int(rng.integers(1, 5)))
    cfg, W, d = build(tmp_path, layers, seed=400 + seed, width=int(rng.choice([64, 96, 192])), vocab=int(rng.choice([64, 250])))
    t = toks(300, cfg["vocab"], seed)
    want = oracle_for(cfg, W).forward(t)
    with open_engine(d) as e:
        close32(feed_whole(e, t), want, 4)
    with open_engine(d, dtype="bfloat16") as e:
        close16(feed_whole(e, t), want, 0.8)
        close16(feed_portions(e, t, [130, 70, 33, 12, 2, 1]), want, 0.8)


# ---------------------------------------------------------------- the engine's own generation path
def greedy_agrees(o, prompt, got):
    want, margin = o.generate(prompt, len(got))
    if margin > 1e-3:
        assert got == want
    else:      # a tie within fp32 rounding may go either way: agree up to the first close call
        k = 0
        while k < len(got) and got[k] == want[k]:
            k += 1
        assert k >= 1


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_submit_scheduler_and_sampler(mix, dtype):
    """More requests than slots, a token budget that cuts prompts into portions, generation by the engine's argmax."""
    cfg, W, d, o = mix
    prompts = [toks(n, cfg["vocab"], 40 + i) for i, n in enumerate((37, 5, 21, 50, 2))]
    with open_engine(d, dtype=dtype, max_tokens=96, max_seqs=2, budget=16, blocks=12) as e:
        outs = e.generate(prompts, max_tokens=12)
        st = e.stats()
    assert st.kv_blocks_free == 12
    for p, got in zip(prompts, outs):
        assert len(got) == 12
        if dtype == "float32":
            greedy_agrees(o, p, got)
        else:
            row = np.sort(o.forward(p)[-1])
            if row[-1] - row[-2] > 1.0:
                assert got[0] == int(np.argmax(o.forward(p)[-1]))


def test_preemption_recomputes_cache_and_state_from_the_start(wide):
    """A pool too small for all running sequences to finish: the scheduler preempts and recomputes; outputs do not change."""
    cfg, W, d, o = wide
    prompts = [toks(n, cfg["vocab"], 60 + i) for i, n in enumerate((30, 28, 31))]
    with open_engine(d, max_tokens=64, max_seqs=3, budget=64, blocks=8) as e:
        outs = e.generate(prompts, max_tokens=20)
        assert e.stats().preemptions > 0
    for p, got in zip(prompts, outs):
        greedy_agrees(o, p, got)


def test_chat_completion_through_the_serving_shell(tmp_path):
    """The design behind the HTTP handler chain, stepped by the engine's own background loop: prompt rendering, submit,
    continuous batching of two concurrent requests, greedy sampling, SSE framing; the tokens are the oracle's."""
    import json
    import threading
    from kubeai_b200.engine import Engine, default_config
    from kubeai_b200.server import Server, tokenize
    V = 300
    cfg, W, d = build(tmp_path, [attention(), delta(), attention(window=40, mlp=None)], seed=51, vocab=V)
    o = oracle_for(cfg, W)
    lim = default_config(manual_step=0, enable_prefix_caching=0, max_num_seqs=4, max_batched_tokens=32, max_model_len=256, num_kv_blocks=64)
    eng = Engine(lim, d, dtype="float32")
    srv = Server([eng], model="db", vocab=V, max_model_len=256)
    try:
        out = {}

        def ask(i, text):
            body = dict(model="db", messages=[{"role": "user", "content": text}], max_tokens=5, temperature=0, stream=(i == 0))
            out[i] = srv.handle("POST", "/openai/v1/chat/completions", json.dumps(body))

        th = [threading.Thread(target=ask, args=(i, t)) for i, t in enumerate(["Hello there, how are you?", "Hi"])]
        for t in th:
            t.start()
        for t in th:
            t.join()
        assert out[0].status == 200 and out[1].status == 200
        ev = out[0].sse_events()
        assert ev[-1] == "[DONE]"
        text0 = "".join(json.loads(e)["choices"][0]["delta"].get("content", "") for e in ev[:-1] if json.loads(e)["choices"])
        text1 = out[1].json()["choices"][0]["message"]["content"]
        for text, user in ((text0, "Hello there, how are you?"), (text1, "Hi")):
            prompt = srv.render_prompt("/v1/chat/completions", json.dumps(dict(model="db", messages=[{"role": "user", "content": user}])))
            got = tokenize(text, V)
            assert len(got) == 5
            greedy_agrees(o, prompt, got)
    finally:
        srv.close()
        eng.close()


def test_a_checkpoint_that_does_not_fit_the_config_is_refused(tmp_path):
    from kubeai_b200 import B200Error
    from kubeai_b200.engine import Engine, default_config
    cfg = make_config([attention(), delta(), attention(mlp=moe(shared=0))])
    for i, name in enumerate(["l0.mix.sink", "l0.mix.k.norm", "l1.mix.A_log", "l1.mix.v.conv", "l1.mlp.correction", "l1.mlp.e5.down", "embed.norm", "final.norm", "l2.norm2"]):
        short = random_weights(cfg)
        if i % 2:
            del short[name]
        else:
            short[name] = np.zeros(int(short[name].size) + 1, dtype=np.float32)
        with pytest.raises(B200Error, match=name):
            Engine(default_config(manual_step=1), write_model_dir(tmp_path / ("c%d" % i), cfg, short), dtype="float32")
