"""Soselix through the engine against the plain oracle (oracle/soselix_oracle.py): each mechanism alone, prefill against
token-by-token decoding, portions down to two tokens, unequal batches, pages and slots used again, far keys found by a
planted query/key pair (at page borders, in prompts and in decoding), a shared latent cache, the sink, far tokens in both
recurrent states, the carried inputs of the convolution across cuts, other sizes (also the degenerate ones), long decoding,
and greedy generation through the engine's own submit / scheduler / sampling path.  Configurations and weights are made
here; nothing is read from disk but what the test wrote."""
import numpy as np
import pytest

from soselix_util import (bf16_round, dense, feed_portions, feed_whole, hgrn2, latent, make_config, mamba2, open_engine, oracle_for, plant_pair,
                          random_weights, rel_err, write_model_dir)

pytestmark = pytest.mark.gpu

F32_TOL = 2e-5     # fp32 engine vs float64 oracle, relative RMS over the vocabulary


def close32(got, want, scale=1.0):
    r = rel_err(got, want)
    assert np.median(r) < F32_TOL * scale, np.median(r)
    assert r.max() < 15 * F32_TOL * scale, (int(np.argmax(r)), r.max())


def close16(got, want):
    """bf16 serving precision on these tiny widths: a percent or two per row; where two keys' scores nearly tie under a sharp
    softmax, or a head's output nearly cancels in front of its norm, rounding may move a single row further."""
    r = rel_err(got, want)
    assert np.median(r) < 0.03, np.median(r)
    assert np.quantile(r, 0.95) < 0.12, np.quantile(r, 0.95)


def toks(n, vocab, seed=0):
    return np.random.default_rng(seed).integers(0, vocab, size=n).tolist()


def build(tmp_path, layers, seed=0, wkw=None, edit=None, **kw):
    cfg = make_config(layers, **kw)
    W = random_weights(cfg, seed=seed, **(wkw or {}))
    if edit:
        edit(W)
    return cfg, W, write_model_dir(tmp_path / "m", cfg, W)


# every kind of layer, with and without a feed-forward, two layers that read layer 0's latents
MIX = [latent(), mamba2(mlp=None), latent(heads=2, dim=5, vdim=7, q_rank=6, kv_from=0), hgrn2(),
       latent(heads=1, dim=8, rot_dim=6, vdim=4, kv_rank=7, q_rank=11, base=3000.0, mlp=None), mamba2(heads=3, vdim=4, state=6, groups=1, norm_groups=2, conv=4),
       latent(heads=4, kv_from=0, scale=0.5, mlp=None)]


@pytest.fixture(scope="module")
def mix(tmp_path_factory):
    cfg, W, d = build(tmp_path_factory.mktemp("mix"), MIX)
    return cfg, W, d, oracle_for(cfg, W)


# ---------------------------------------------------------------- each mechanism alone
def zero(*names):
    def edit(W):
        for n in names:
            W[n][...] = 0.0
    return edit


@pytest.mark.parametrize("name,layers,kw,edit", [
    ("latent_only", [latent(mlp=None)], {}, None),
    ("latent_one_head", [latent(heads=1, dim=3, vdim=2, kv_rank=5, q_rank=1, mlp=None)], {}, None),
    ("latent_rotated_scores_alone", [latent(scale=1.0, mlp=None)], {}, zero("l0.mix.uk")),
    ("latent_unrotated_scores_alone", [latent(mlp=None)], {}, lambda W: W["l0.mix.dkv"][10:].fill(0.0)),
    ("latent_two_rotated_dims", [latent(rot_dim=2, base=7.0, mlp=None)], {}, None),
    ("latent_many_heads", [latent(heads=19, dim=4, vdim=3, kv_rank=8, rot_dim=8, mlp=None)], {}, None),
    ("latent_value_wider_than_rank", [latent(heads=2, vdim=13, kv_rank=6, q_rank=30, mlp=None)], {}, None),
    ("latent_shared_by_the_next_layer", [latent(mlp=None), latent(heads=5, dim=2, vdim=3, q_rank=4, scale=0.7, kv_from=0, mlp=None)], {}, None),
    ("latent_shared_by_two_later_layers", [hgrn2(mlp=None), latent(), mamba2(), latent(kv_from=1, mlp=None), latent(heads=2, kv_from=1)], {}, None),
    ("latent_two_caches", [latent(), latent(kv_rank=6, rot_dim=8), latent(kv_from=0), latent(kv_rank=6, rot_dim=8, kv_from=1)], {}, None),
    ("hgrn2_only", [hgrn2(mlp=None)], {}, None),
    ("hgrn2_one_channel", [hgrn2(heads=3, dim=1, vdim=1, mlp=None)], {}, None),
    ("hgrn2_many_rows", [hgrn2(heads=2, dim=70, vdim=9, mlp=None)], {}, None),
    ("hgrn2_wide_value", [hgrn2(heads=1, dim=4, vdim=150, mlp=None)], {}, None),
    ("hgrn2_no_lower_bound", [hgrn2(mlp=None)], {}, zero("l0.mix.lower")),
    ("mamba2_only", [mamba2(mlp=None)], {}, None),
    ("mamba2_one_head", [mamba2(heads=1, vdim=5, state=3, groups=1, norm_groups=1, conv=2, mlp=None)], {}, None),
    ("mamba2_a_group_per_head", [mamba2(heads=4, groups=4, norm_groups=4, mlp=None)], {}, None),
    ("mamba2_one_group_many_heads", [mamba2(heads=6, groups=1, norm_groups=1, mlp=None)], {}, None),
    ("mamba2_norm_groups_across_heads", [mamba2(heads=4, vdim=6, norm_groups=8, mlp=None)], {}, None),
    ("mamba2_one_state", [mamba2(state=1, mlp=None)], {}, None),
    ("mamba2_wide_state", [mamba2(heads=2, vdim=3, state=100, norm_groups=1, mlp=None)], {}, None),
    ("mamba2_one_tap", [mamba2(conv=1, mlp=None)], {}, None),
    ("mamba2_six_taps", [mamba2(conv=6, mlp=None)], {}, None),
    ("mamba2_without_skip", [mamba2(mlp=None)], {}, zero("l0.mix.D")),
    ("mamba2_skip_alone", [mamba2(mlp=None)], {}, lambda W: W["l0.mix.dt_bias"].fill(-60.0)),
    ("mamba2_large_steps", [mamba2(mlp=None)], {}, lambda W: W["l0.mix.dt_bias"].fill(24.0)),
    ("feed_forward", [hgrn2(mlp=dense(31))], {}, None),
    ("feed_forward_of_one", [hgrn2(mlp=dense(1))], {}, None),
    ("feed_forward_unequal_curves", [mamba2(mlp=dense(20))], {}, lambda W: W["l0.mlp.act"].__setitem__(slice(None), [2.0, -3.0])),
    ("plain_residual", [latent(), hgrn2(), mamba2()], dict(mult=1.0, embed=1.0), None),
    ("odd_width", [latent(), hgrn2(), mamba2(), latent(kv_from=0)], dict(width=21, vocab=33), None),
    ("large_eps_in_every_norm", [latent(), hgrn2(), mamba2(), latent(kv_from=0)], dict(eps=0.05), None),
])
def test_each_mechanism_matches_the_oracle(tmp_path, name, layers, kw, edit):
    cfg, W, d = build(tmp_path, layers, seed=3, edit=edit, **kw)
    o = oracle_for(cfg, W)
    t = toks(29, cfg["vocab"], 1)
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
    """The query latent's and the hidden layer's size may stand in the checkpoint alone."""
    import json
    cfg, W, d = build(tmp_path, [latent(q_rank=13), hgrn2(mlp=dense(11))], seed=4)
    short = json.loads(json.dumps(cfg))
    del short["layers"][0]["mixer"]["q_rank"]
    del short["layers"][1]["mlp"]["ff"]
    t = toks(20, cfg["vocab"], 1)
    with open_engine(write_model_dir(tmp_path / "s", short, W)) as e:
        close32(feed_whole(e, t), oracle_for(cfg, W).forward(t))


def test_bfloat16_serving_precision_stays_near_the_oracle(mix):
    cfg, W, d, o = mix
    t = toks(70, cfg["vocab"], 2)
    want = o.forward(t)
    with open_engine(d, dtype="bfloat16") as e:
        close16(feed_whole(e, t), want)
        close16(feed_portions(e, t, [40, 1]), want)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seqs", [1, 5, 12, 17])
def test_decode_batches_of_every_width(tmp_path, dtype, seqs):
    """Steps of one token per sequence at batch sizes on both sides of the few-row product kernels' limits, at sizes that
    are multiples of 8 (the vector paths) with inner sizes that do not fill a whole k-step; fp32 results per row must not
    depend on the batch."""
    layers = [latent(heads=4, dim=24, rot_dim=16, vdim=40, kv_rank=48, q_rank=56), hgrn2(heads=2, dim=24, vdim=40, mlp=dense(264)),
              mamba2(heads=4, vdim=24, state=16, groups=2, norm_groups=4, conv=4, mlp=dense(88)), latent(heads=2, dim=40, rot_dim=16, vdim=24, kv_rank=48, q_rank=72, kv_from=0)]
    cfg, W, d = build(tmp_path, layers, seed=19, width=88, vocab=100)
    o = oracle_for(cfg, W)
    ts = [toks(9, 100, 20 + i) for i in range(seqs)]
    with open_engine(d, dtype=dtype, max_tokens=64, max_seqs=seqs, budget=256) as e:
        rids = [e.feed_open() for _ in ts]
        e.feed_step([(r, t[:4], []) for r, t in zip(rids, ts)])
        got = [e.feed_step([(r, [t[k]], [0]) for r, t in zip(rids, ts)]) for k in range(4, 9)]
        for r in rids:
            e.feed_close(r)
    want = np.stack([o.forward(t)[4:] for t in ts], axis=1)
    (close32 if dtype == "float32" else close16)(np.concatenate(got), want.reshape(-1, 100))


def test_bfloat16_widths_the_tensor_core_projection_cannot_take(tmp_path):
    """A width and inner sizes that are no multiple of 8 run on the general linear kernels."""
    layers = [latent(heads=3, dim=5, vdim=3), hgrn2(heads=3, dim=5, vdim=3, mlp=dense(7)), mamba2(heads=3, vdim=5, state=3, groups=3, norm_groups=1), latent(kv_from=0)]
    cfg, W, d = build(tmp_path, layers, width=20, vocab=33)
    t = toks(40, 33, 4)
    want = oracle_for(cfg, W).forward(t)
    with open_engine(d, dtype="bfloat16") as e:
        close16(feed_whole(e, t), want)
        close16(feed_portions(e, t, [20, 3, 1]), want)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_medium_sizes_on_every_projection_path(tmp_path, dtype):
    layers = [latent(heads=4, dim=16, rot_dim=16, vdim=24, kv_rank=32, q_rank=40, mlp=dense(104)), hgrn2(heads=3, dim=40, vdim=24, mlp=dense(512)),
              mamba2(heads=8, vdim=16, state=24, groups=4, norm_groups=2, conv=4, mlp=dense(256)), latent(heads=2, dim=24, rot_dim=16, vdim=40, kv_rank=32, q_rank=24, kv_from=0)]
    cfg, W, d = build(tmp_path, layers, seed=17, width=72, vocab=90)
    t = toks(300, 90, 18)
    want = oracle_for(cfg, W).forward(t)
    with open_engine(d, dtype=dtype) as e:
        whole = feed_whole(e, t)
        parts = feed_portions(e, t, [140, 9, 33, 16, 1])
    (close32 if dtype == "float32" else close16)(whole, want)
    (close32 if dtype == "float32" else close16)(parts, want)


@pytest.mark.parametrize("heads,kv_rank,rot_dim", [(3, 32, 16), (16, 64, 32), (20, 48, 16), (6, 128, 64), (1, 16, 16), (9, 512, 64)])
def test_bfloat16_tensor_core_attention_equals_the_general_kernel(tmp_path, monkeypatch, heads, kv_rank, rot_dim):
    """Latent widths that fit the mma fragments: the 16-, 32- and 64-row kernels and the split form with its merge, all with
    a sink per head and the output gate, against the general kernel on the same bf16 cache; several key tiles, several
    tokens per row tile (few heads), several head groups (more than 16 heads), a shared cache, portions and decoding."""
    layers = [latent(heads=heads, dim=8, rot_dim=rot_dim, vdim=8, kv_rank=kv_rank, q_rank=24, mlp=None),
              latent(heads=heads, dim=8, rot_dim=rot_dim, vdim=8, kv_rank=kv_rank, q_rank=16, kv_from=0, mlp=None)]
    cfg, W, d = build(tmp_path, layers, seed=21, width=32, wkw=dict(sink=(2.0, 1.5)))
    t = toks(230, cfg["vocab"], 22)
    want = oracle_for(cfg, W).forward(t)
    cuts = [67, 2, 90, 1]
    out = {}
    for name, env in (("default", {}), ("general", dict(B200_NX_ATTN_MMA="0")), ("split", dict(B200_NX_ATTN_SPLIT="3")), ("wide", dict(B200_NX_ATTN_WIDE="1"))):
        for k, v in env.items():
            monkeypatch.setenv(k, v)
        with open_engine(d, dtype="bfloat16") as e:
            out[name] = (feed_whole(e, t), feed_portions(e, t, cuts))
        for k in env:
            monkeypatch.delenv(k)
    for name, pair in out.items():
        for got, plain in zip(pair, out["general"]):
            close16(got, want)
            r = rel_err(got, plain.astype(np.float64))
            assert np.median(r) < 0.02 and r.max() < 0.1, name


def test_bfloat16_large_prompt_step_takes_the_64_row_attention_kernel_by_itself(tmp_path, monkeypatch):
    layers = [latent(heads=16, dim=8, rot_dim=16, vdim=8, kv_rank=48, q_rank=24, mlp=None)]
    cfg, W, d = build(tmp_path, layers, seed=23, width=32, wkw=dict(sink=(2.0, 1.5)))
    seqs = [toks(330, cfg["vocab"], 24 + i) for i in range(2)]
    o = oracle_for(cfg, W)
    want = np.concatenate([o.forward(t) for t in seqs])

    def both():
        with open_engine(d, dtype="bfloat16", max_tokens=1024, max_seqs=2) as e:
            rids = [e.feed_open() for _ in seqs]
            out = e.feed_step([(r, t, list(range(len(t)))) for r, t in zip(rids, seqs)])
            for r in rids:
                e.feed_close(r)
            return out

    got = both()
    monkeypatch.setenv("B200_NX_ATTN_MMA", "0")
    plain = both()
    close16(got, want)
    assert np.median(rel_err(got, plain.astype(np.float64))) < 0.02 and rel_err(got, plain.astype(np.float64)).max() < 0.1


def test_fused_large_step_products_equal_the_plain_ones(tmp_path, monkeypatch):
    """Matrices of whole 256-row tiles in a step with a tile per CTA pair and more take the fused GEMM form: bias and xIELU in
    the epilogue of a wide up-projection, 256-token tiles for a deep down-projection, the filled-up input projection.  The
    step's last token tiles are partial.  Rows of the first tokens are the oracle's; all rows are those of the plain form."""
    layers = [hgrn2(heads=4, dim=96, vdim=104, mlp=dense(4352)), mamba2(heads=8, vdim=120, state=16, groups=1, norm_groups=4, conv=4, mlp=None)]
    cfg, W, d = build(tmp_path, layers, seed=81, width=2048, vocab=64)
    T = 4700
    t = toks(T, 64, 82)
    rows = sorted(set(range(24)) | set(range(100, T, 97)) | {255, 256, 511, 512, 4095, 4096, 4607, 4608, T - 1})
    out = {}
    for knob in ("1", "0"):
        monkeypatch.setenv("B200_SX_FUSE", knob)
        with open_engine(d, dtype="bfloat16", max_tokens=4704, max_seqs=1) as e:
            out[knob] = feed_whole(e, t, rows)
    close16(out["1"][:24], oracle_for(cfg, W).forward(t[:24]))
    r = rel_err(out["1"], out["0"].astype(np.float64))
    assert np.median(r) < 0.01 and r.max() < 0.05, (np.median(r), r.max())


@pytest.mark.parametrize("heads,vdim,state,groups,norm_groups", [(4, 16, 16, 2, 2), (3, 64, 128, 1, 1), (6, 24, 48, 3, 2), (2, 136, 64, 1, 4), (8, 8, 112, 2, 1), (5, 72, 32, 5, 5)])
def test_chunked_tensor_core_scan_equals_the_token_by_token_scan(tmp_path, monkeypatch, heads, vdim, state, groups, norm_groups):
    """State and value sizes that the chunked form of the Mamba-2 recurrence takes (whole and partial blocks of state rows and
    value columns, several chunks of 64, portions that end inside a chunk): it keeps fp32 precision, so only the rounding of
    the layer's bf16 output can differ from the sequential scan."""
    cfg, W, d = build(tmp_path, [mamba2(heads=heads, vdim=vdim, state=state, groups=groups, norm_groups=norm_groups, conv=4, mlp=None)], seed=5, width=64, vocab=60)
    t = toks(333, 60, 6)
    want = oracle_for(cfg, W).forward(t)
    out = {}
    for knob in ("1", "0"):          # from one token per portion; never
        monkeypatch.setenv("B200_SCAN_CHUNK", knob)
        with open_engine(d, dtype="bfloat16") as e:
            out[knob] = (feed_whole(e, t), feed_portions(e, t, [100, 64, 1, 17, 2, 90, 1]))
    for a, b in zip(out["1"], out["0"]):
        close16(a, want)
        r = rel_err(a, b.astype(np.float64))
        assert np.median(r) < 1e-3 and r.max() < 0.01, (np.median(r), r.max())


@pytest.mark.parametrize("rate,step", [(3.0, 6.0), (-7.0, -2.0), (0.0, -60.0)])
def test_chunked_scan_at_extreme_decays(tmp_path, monkeypatch, rate, step):
    """Decays that leave nothing of a state after one token (no factor may overflow), decays next to one, and step sizes of
    zero."""
    cfg, W, d = build(tmp_path, [mamba2(heads=4, vdim=16, state=32, groups=2, norm_groups=2, mlp=None)], seed=7, width=48, vocab=60,
                      edit=lambda W: (W["l0.mix.A_log"].fill(rate), W["l0.mix.dt_bias"].fill(step)))
    t = toks(200, 60, 8)
    want = oracle_for(cfg, W).forward(t)
    with open_engine(d, dtype="bfloat16") as e:
        got = feed_whole(e, t)
    monkeypatch.setenv("B200_SCAN_CHUNK", "0")
    with open_engine(d, dtype="bfloat16") as e:
        one = feed_whole(e, t)
    assert np.isfinite(got).all()
    close16(got, want)
    assert rel_err(got, one.astype(np.float64)).max() < 0.02


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
    cfg, W, d = build(tmp_path, [mamba2(conv=taps, mlp=None), mamba2(heads=2, conv=taps, vdim=12, mlp=None)], seed=6)
    t = toks(33, cfg["vocab"], 7)
    want = oracle_for(cfg, W).forward(t)
    with open_engine(d) as e:
        close32(feed_portions(e, t, [1, 2, 1, 1, 2, 5, 1, 2, 2, 1]), want)
        close32(feed_portions(e, t, [taps - 1, taps, 1, taps + 1, 2]), want)


def test_long_decoding_stays_on_the_oracle(tmp_path):
    cfg, W, d = build(tmp_path, [latent(), mamba2(mlp=None), hgrn2(mlp=None), latent(kv_from=0)], seed=8, wkw=dict(lower=(0.8, 0.99)))
    t = toks(260, cfg["vocab"], 7)
    want = oracle_for(cfg, W).forward(t)
    with open_engine(d) as e:
        got = feed_portions(e, t, [20, 1])
    close32(got, want, 5)


def test_contexts_longer_than_one_round_of_the_general_attention_kernel(tmp_path):
    """The general kernel walks the keys in rounds of 1024 with a running maximum: a prompt of 2100 tokens crosses two
    borders, and the last rows of a decode step sit behind them."""
    cfg, W, d = build(tmp_path, [latent(heads=2, mlp=None)], seed=9, width=16, vocab=30, wkw=dict(sink=(1.0, 0.5)))
    t = toks(2100, 30, 10)
    want = oracle_for(cfg, W).forward(t)
    with open_engine(d, max_tokens=2112, max_seqs=1) as e:
        r = e.feed_open()
        a = e.feed_step([(r, t[:2090], list(range(0, 2090, 7)) + [1023, 1024, 1025, 2047, 2048, 2049])])
        b = np.concatenate([e.feed_step([(r, [x], [0])]) for x in t[2090:]])
        e.feed_close(r)
    close32(a, want[list(range(0, 2090, 7)) + [1023, 1024, 1025, 2047, 2048, 2049]], 2)
    close32(b, want[2090:], 2)


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
    layers = [latent(heads=4, dim=16, rot_dim=16, vdim=16, kv_rank=32, q_rank=32, mlp=dense(64)), mamba2(heads=4, vdim=16, state=16, norm_groups=2, mlp=None),
              latent(heads=8, dim=8, rot_dim=16, vdim=8, kv_rank=32, q_rank=16, kv_from=0, mlp=None), hgrn2(heads=2, dim=16, vdim=16, mlp=dense(64))]
    cfg, W, d = build(tmp_path, layers, seed=71, width=32)
    o = oracle_for(cfg, W)
    seqs = [toks(n, cfg["vocab"], 72 + i) for i, n in enumerate((150, 61, 9, 120))]
    plan = [(70, 1, 9, 33), (37, 1, 0, 2), (1, 40, 0, 64), (42, 1, 0, 1), (0, 18, 0, 20)]
    with open_engine(d, dtype="bfloat16", max_tokens=160) as e:
        got = run_plan(e, seqs, plan)
        alone = [feed_whole(e, t) for t in seqs]
    for i in range(4):
        close16(got[i], o.forward(seqs[i]))
        assert np.median(rel_err(got[i], alone[i].astype(np.float64))) < 0.02 and rel_err(got[i], alone[i].astype(np.float64)).max() < 0.1


def feed_portions_on(e, r, tokens, sizes):
    outs, at, i = [], 0, 0
    while at < len(tokens):
        n = min(sizes[min(i, len(sizes) - 1)], len(tokens) - at)
        outs.append(e.feed_step([(r, tokens[at:at + n], list(range(n)))]))
        at += n
        i += 1
    e.feed_close(r)
    return np.concatenate(outs)


def test_pages_and_slots_are_used_again(mix):
    """A pool of exactly two sequences' pages and two slots: later requests run in what earlier ones gave back, and start
    from empty states and empty carried inputs whatever the slot held."""
    cfg, W, d, o = mix
    seqs = [toks(n, cfg["vocab"], 20 + i) for i, n in enumerate((40, 33, 48, 17, 41))]
    with open_engine(d, max_tokens=48, max_seqs=2, blocks=6, budget=96) as e:
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
    close32(got_c, o.forward(seqs[2]))
    close32(got_f, o.forward(seqs[3]))
    close32(got_g, o.forward(seqs[4]))


def test_a_step_over_the_pool_is_refused_and_leaves_the_engine_usable(mix):
    from kubeai_b200 import B200Error
    cfg, W, d, o = mix
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


def test_a_model_without_attention_and_one_without_recurrence(tmp_path):
    for i, layers in enumerate(([hgrn2(), mamba2()], [latent(), latent(kv_from=0)])):
        cfg, W, d = build(tmp_path / str(i), layers, seed=33 + i)
        o = oracle_for(cfg, W)
        seqs = [toks(n, cfg["vocab"], 34 + k) for k, n in enumerate((30, 12))]
        with open_engine(d, max_tokens=64, max_seqs=2) as e:
            got = run_plan(e, seqs, [(9, 1), (1, 3), (20, 0)])
        for k in range(2):
            close32(got[k], o.forward(seqs[k]))


# ---------------------------------------------------------------- far keys made visible
QTOK, KTOK = 7, 11


@pytest.fixture(scope="module")
def planted(tmp_path_factory):
    """One attention layer that copies from KTOK positions whenever a QTOK position can see one (planted pair, sharp
    softmax against a sink that would otherwise win, rotated parts off), and a second one on the same latents."""
    cfg = make_config([latent(heads=2, dim=12, rot_dim=16, vdim=10, kv_rank=16, q_rank=20, scale=3.0, mlp=None),
                       latent(heads=1, dim=6, rot_dim=16, vdim=8, kv_rank=16, q_rank=8, kv_from=0, mlp=None)], width=48, vocab=40)
    W = plant_pair(cfg, random_weights(cfg, seed=31, sink=(3.0, 0.2)), QTOK, KTOK)
    return cfg, W, write_model_dir(tmp_path_factory.mktemp("planted") / "m", cfg, W), oracle_for(cfg, W)


def sequence_with(n, marks, seed):
    """Random filler without the two special tokens, marks[position] = token."""
    t = np.random.default_rng(seed).integers(12, 40, size=n).tolist()
    for p, x in marks.items():
        t[p] = x
    return t


@pytest.mark.parametrize("key,query", [(0, 15), (0, 16), (15, 16), (16, 17), (31, 400), (0, 447), (63, 64), (64, 128), (127, 130), (255, 440), (1, 2)])
def test_a_far_key_is_found_wherever_it_lies(planted, key, query):
    """First positions, page borders, tile borders, hundreds of positions apart; in a prompt, in portions cut between key
    and query or around the query, and decoded."""
    cfg, W, d, o = planted
    n = query + 3
    t = sequence_with(n, {key: KTOK, query: QTOK}, 1)
    gone = list(t)
    gone[key] = 13
    want = o.forward(t)
    assert rel_err(want[query:query + 1], o.forward(gone)[query:query + 1])[0] > 0.3      # the key decides
    with open_engine(d) as e:
        close32(feed_whole(e, t), want)
        close32(feed_portions(e, t, [key + 1, max(1, query - key - 1), 1]), want)
        close32(feed_portions(e, t, [query, 1]), want)
        close32(feed_portions(e, t, [max(1, query - 1), 2, 1]), want)
    with open_engine(d, dtype="bfloat16") as e:
        for got in (feed_whole(e, t), feed_portions(e, t, [query, 1])):
            r = rel_err(got, want)
            assert np.median(r) < 0.05 and r[query] < 0.2


@pytest.mark.parametrize("query", [15, 16, 31, 63, 64, 200])
def test_a_key_behind_the_query_is_not_seen(planted, query):
    """The token after the query (in the same step, page or tile) would decide its logits if it were visible."""
    cfg, W, d, o = planted
    t = sequence_with(query + 6, {query: QTOK, query + 1: KTOK, query + 2: KTOK}, 2)
    plain = list(t)
    plain[query + 1], plain[query + 2] = 14, 15
    want = o.forward(t)
    with open_engine(d) as e:
        a, b = feed_whole(e, t), feed_whole(e, plain)
        assert np.abs(a[query] - b[query]).max() < 1e-4 * np.abs(a[query]).max()
        close32(a, want)
        close32(feed_portions(e, t, [query + 1, 2, 1]), want)
    with open_engine(d, dtype="bfloat16") as e:
        assert np.median(rel_err(feed_whole(e, t), want)) < 0.05
        assert rel_err(feed_whole(e, t), want)[query] < 0.2


def test_a_far_key_survives_other_requests_in_the_batch(planted):
    cfg, W, d, o = planted
    a = sequence_with(200, {3: KTOK, 197: QTOK}, 5)
    b = sequence_with(90, {60: KTOK, 88: QTOK}, 6)
    c = sequence_with(70, {69: QTOK}, 7)          # no key of its own: it must not find the others'
    with open_engine(d, max_tokens=208) as e:
        got = run_plan(e, [a, b, c], [(100, 30, 2), (33, 1, 30), (60, 55, 30), (3, 1, 5)])
    for g, t in zip(got, (a, b, c)):
        close32(g, o.forward(t))


def test_the_sink_takes_its_share_of_the_softmax(tmp_path):
    """A large sink empties the attention, a very negative one leaves the plain softmax: both follow the oracle, and differ;
    so do sinks that differ from head to head."""
    cfg = make_config([latent(heads=2, dim=8, rot_dim=16, vdim=8, kv_rank=16, mlp=None)])
    W = random_weights(cfg, seed=15)
    t = toks(90, cfg["vocab"], 16)
    outs = []
    for i, sink in enumerate(([6.0, 6.0], [-30.0, -30.0], [6.0, -30.0], [90.0, -1e4])):
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
    assert min(rel_err(a, b).max() for k, a in enumerate(outs) for b in outs[k + 1:]) > 0.05


def test_distance_turns_the_rotated_scores(tmp_path):
    """With the unrotated scores off only the distance of the key counts: positions far into a sequence still see the right
    angles, in a prompt and behind cuts."""
    cfg, W, d = build(tmp_path, [latent(rot_dim=8, base=50000.0, scale=2.0, mlp=None)], seed=25, edit=lambda W: W["l0.mix.uk"].fill(0.0))
    t = toks(420, cfg["vocab"], 26)
    want = oracle_for(cfg, W).forward(t)
    with open_engine(d) as e:
        close32(feed_whole(e, t), want, 2)
        close32(feed_portions(e, t, [333, 40, 1]), want, 2)


# ---------------------------------------------------------------- far tokens in the recurrent states
@pytest.mark.parametrize("kind", ["hgrn2", "mamba2"])
def test_far_tokens_reach_through_the_state(tmp_path, kind):
    """With gates close to one the state carries the first tokens across hundreds of positions: other first tokens change
    the last logits, and the engine follows the oracle whether the prompt comes whole, in portions or decoded."""
    if kind == "hgrn2":
        layers, edit = [hgrn2(heads=2, dim=8, vdim=8, mlp=None)], lambda W: W["l0.mix.lower"].fill(0.99609375)
    else:
        layers, edit = [mamba2(mlp=None)], lambda W: (W["l0.mix.A_log"].fill(-7.0), W["l0.mix.dt_bias"].fill(-2.0))
    cfg, W, d = build(tmp_path, layers, seed=41, edit=edit)
    o = oracle_for(cfg, W)
    a = toks(300, cfg["vocab"], 42)
    b = [(x + 1) % cfg["vocab"] for x in a[:20]] + a[20:]
    wa, wb = o.forward(a), o.forward(b)
    assert rel_err(wa[-1:], wb[-1:])[0] > 0.01
    with open_engine(d) as e:
        close32(feed_whole(e, a), wa, 3)
        close32(feed_portions(e, b, [150, 33, 1]), wb, 3)
    with open_engine(d, dtype="bfloat16") as e:
        close16(feed_whole(e, a), wa)


def test_the_write_of_a_nearly_closed_forget_gate_keeps_its_digits(tmp_path):
    """Gates so near one that f itself rounds to 1 in fp32 still write (1 - f) v: the complement is formed on its own.  With
    every gate like that the normed output depends on those small writes alone."""
    cfg, W, d = build(tmp_path, [hgrn2(heads=1, dim=6, vdim=6, mlp=None)], seed=43, eps=1e-30,
                      edit=lambda W: (W["l0.mix.f.b"].fill(18.0), W["l0.mix.lower"].fill(0.0)))
    t = toks(40, cfg["vocab"], 44)
    with open_engine(d) as e:
        close32(feed_whole(e, t), oracle_for(cfg, W).forward(t), 5)


def test_first_tokens_of_a_sequence(mix):
    cfg, W, d, o = mix
    with open_engine(d) as e:
        for n in (1, 2, 3):
            t = toks(n, cfg["vocab"], 50 + n)
            close32(feed_whole(e, t), o.forward(t))
        t = toks(6, cfg["vocab"], 54)
        close32(feed_portions(e, t, [1, 1, 2]), o.forward(t))


def random_layers(rng, n, pick_size):
    """n layers in random order; an attention layer may read the latents of an earlier one that has its own."""
    layers, own = [], []
    for i in range(n):
        mlp = None if rng.random() < 0.3 else dense(pick_size(30))
        k = int(rng.integers(0, 3))
        if k == 0:
            if own and rng.random() < 0.5:
                j = own[int(rng.integers(0, len(own)))]
                src = layers[j]["mixer"]
                layers.append(latent(heads=int(rng.integers(1, 6)), dim=pick_size(9), rot_dim=src["rot_dim"], vdim=pick_size(9), kv_rank=src["kv_rank"],
                                     q_rank=pick_size(14), base=src["rot"]["base"], scale=float(rng.uniform(0.1, 0.6)), kv_from=j, mlp=mlp))
            else:
                own.append(i)
                layers.append(latent(heads=int(rng.integers(1, 6)), dim=pick_size(9), rot_dim=2 * pick_size(5), vdim=pick_size(9), kv_rank=pick_size(16),
                                     q_rank=pick_size(14), base=float(rng.choice([30.0, 1e4, 5e5])), scale=float(rng.uniform(0.1, 0.6)), mlp=mlp))
        elif k == 1:
            layers.append(hgrn2(heads=int(rng.integers(1, 4)), dim=pick_size(20), vdim=pick_size(20), mlp=mlp))
        else:
            G, Hg, Dv = int(rng.integers(1, 4)), int(rng.integers(1, 4)), pick_size(12)
            inner = G * Hg * Dv
            layers.append(mamba2(heads=G * Hg, vdim=Dv, state=pick_size(20), groups=G, conv=int(rng.integers(1, 6)),
                                 norm_groups=int(rng.choice([x for x in range(1, inner + 1) if inner % x == 0 and x <= 12])), mlp=mlp))
    return layers


@pytest.mark.parametrize("seed", range(10))
def test_random_configurations(tmp_path, seed):
    rng = np.random.default_rng(100 + seed)
    layers = random_layers(rng, int(rng.integers(1, 6)), lambda hi: int(rng.integers(1, hi)))
    cfg, W, d = build(tmp_path, layers, seed=200 + seed, width=int(rng.integers(6, 40)), vocab=int(rng.integers(5, 60)),
                      mult=float(rng.uniform(0.3, 1.2)), embed=float(rng.uniform(0.5, 4.0)), wkw=dict(lower=(0.0, float(rng.uniform(0.5, 0.99)))))
    t = toks(70, cfg["vocab"], seed)
    want = oracle_for(cfg, W).forward(t)
    with open_engine(d) as e:
        close32(feed_whole(e, t), want, 3)
        close32(feed_portions(e, t, [int(rng.integers(2, 30)), int(rng.integers(1, 9)), 1]), want, 3)


@pytest.mark.parametrize("seed", range(5))
def test_bfloat16_random_medium_configurations(tmp_path, seed):
    """Sizes that the tensor-core projections and the tensor-core attention take (multiples of 16), in random layer orders:
    the bf16 engine stays near the oracle whole and in portions, and the fp32 engine on all rows."""
    rng = np.random.default_rng(300 + seed)
    layers = random_layers(rng, int(rng.integers(3, 6)), lambda hi: 16 * int(rng.integers(1, 5)))
    for ly in layers:
        ly["mixer"]["scale"] = 0.1
        if ly["mlp"]:
            ly["mlp"]["ff"] *= int(rng.choice([1, 4]))
    cfg, W, d = build(tmp_path, layers, seed=400 + seed, width=int(rng.choice([64, 96, 192])), vocab=int(rng.choice([64, 250])), mult=0.5)
    t = toks(300, cfg["vocab"], seed)
    want = oracle_for(cfg, W).forward(t)
    with open_engine(d) as e:
        close32(feed_whole(e, t), want, 3)
    with open_engine(d, dtype="bfloat16") as e:
        close16(feed_whole(e, t), want)
        close16(feed_portions(e, t, [130, 70, 33, 12, 2, 1]), want)


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
            if row[-1] - row[-2] > 0.3:
                assert got[0] == int(np.argmax(o.forward(p)[-1]))


def test_preemption_recomputes_cache_and_state_from_the_start(mix):
    """A pool too small for all running sequences to finish: the scheduler preempts and recomputes; outputs do not change."""
    cfg, W, d, o = mix
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
    cfg, W, d = build(tmp_path, [latent(), mamba2(), hgrn2(mlp=None), latent(kv_from=0)], seed=51, vocab=V)
    o = oracle_for(cfg, W)
    lim = default_config(manual_step=0, enable_prefix_caching=0, max_num_seqs=4, max_batched_tokens=32, max_model_len=256, num_kv_blocks=64)
    eng = Engine(lim, d, dtype="float32")
    srv = Server([eng], model="sx", vocab=V, max_model_len=256)
    try:
        out = {}

        def ask(i, text):
            body = dict(model="sx", messages=[{"role": "user", "content": text}], max_tokens=5, temperature=0, stream=(i == 0))
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
            prompt = srv.render_prompt("/v1/chat/completions", json.dumps(dict(model="sx", messages=[{"role": "user", "content": user}])))
            got = tokenize(text, V)
            assert len(got) == 5
            greedy_agrees(o, prompt, got)
    finally:
        srv.close()
        eng.close()


def test_a_checkpoint_that_does_not_fit_the_config_is_refused(tmp_path):
    from kubeai_b200 import B200Error
    from kubeai_b200.engine import Engine, default_config
    cfg = make_config([latent(), mamba2(), hgrn2(), latent(kv_from=0)])
    for i, name in enumerate(["l0.mix.sink", "l0.mix.dkv.norm", "l1.mix.A_log", "l1.mix.conv.b", "l2.mix.lower", "l3.mix.uq", "l3.mlp.down.b", "final.norm"]):
        short = random_weights(cfg)
        if i % 2:
            del short[name]
        else:
            short[name] = np.zeros(int(short[name].size) + 1, dtype=np.float32)
        with pytest.raises(B200Error, match=name):
            Engine(default_config(manual_step=1), write_model_dir(tmp_path / ("c%d" % i), cfg, short), dtype="float32")
