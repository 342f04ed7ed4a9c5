"""Mizerax on the GPU against the plain restatement in tests/mizerax_oracle.py: every mechanism alone (op-level entry points that launch
the family's kernels), then whole models with small random configurations — prompts in one pass, token by token, in portions, after a
release, long decoding, greedy generation through the host entry points and the command line."""
import json
import math
import os
import subprocess

import numpy as np
import pytest

import mizerax_oracle as O
from xalm_b200 import build, capi
from xalm_b200 import safetensors_io as ST
from xalm_b200.model import InferenceState, Model, Sampler, generate

pytestmark = pytest.mark.gpu

F32_TOL = 2e-4   # IEEE fp32 path against float64, on values of order one
BF16_TOL = 6e-2  # serving mode: bf16 weights (exact here), a bf16 key/value cache, fp16 operands on the tensor cores


def close(got, want, tol):
    got, want = np.asarray(got, dtype=np.float64), np.asarray(want, dtype=np.float64)
    assert got.shape == want.shape, (got.shape, want.shape)
    err = np.abs(got - want).max() / max(1.0, np.abs(want).max())
    assert err < tol, f"max error {err:.3e} (tolerance {tol})"


def rows_within(got, want, tol, share=0.1):
    """16-bit mode: most rows within rounding of the oracle (an expert choice decided by less than 16-bit noise flips, and that token's row is
    off from there on)."""
    err = np.abs(np.asarray(got, dtype=np.float64) - want).max(axis=1) / max(1.0, np.abs(want).max())
    assert np.median(err) < tol / 4 and (err > tol).mean() <= share, f"median {np.median(err):.3e}, over {(err > tol).mean():.2f}"


# ---- mechanisms alone ----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("T,W", [(1, 5), (3, 24), (7, 130), (2, 256), (5, 1000), (2, 4096), (1, 13000)])
def test_layer_norm(T, W):
    """Rows whose mean is far from zero: the deviations must be taken from the mean, not from a difference of large sums; a missing bias."""
    rng = np.random.default_rng(W)
    x = rng.standard_normal((T, W)).astype(np.float32) * 0.5 + 50.0
    w, b = 1 + 0.3 * rng.standard_normal(W), rng.standard_normal(W)
    close(capi.layer_norm(x, w, b, 1e-4), O.layer_norm(x.astype(np.float64), w, b, 1e-4), F32_TOL)
    close(capi.layer_norm(x, w, None, 0.5), O.layer_norm(x.astype(np.float64), w, 0.0, 0.5), F32_TOL)   # an eps that matters


def test_position_rows():
    rng = np.random.default_rng(0)
    w = {"embed": rng.standard_normal((11, 20)), "pos": rng.standard_normal((30, 20))}
    for p0, tokens in ((0, [3, 3, 0]), (27, [10, 1, 5]), (29, [7])):
        close(capi.embed_positions(tokens, p0, w["embed"], w["pos"]), O.embed_rows(w, tokens, p0), 1e-6)
    with pytest.raises(capi.XalmError):
        capi.embed_positions([1, 2], 29, w["embed"], w["pos"])


@pytest.mark.parametrize("H,G,d,dv", [(4, 2, 6, 9), (1, 1, 1, 3), (6, 3, 40, 8), (8, 1, 128, 64)])
@pytest.mark.parametrize("coef,every", [(0.0, 0), (0.6, 1), (0.8, 7), (-0.1, 300)])
def test_head_norms_and_query_temperature(H, G, d, dv, coef, every):
    """Queries, keys and values in one projection row; positions on either side of a temperature step; one loud head (its norm is its own)."""
    rng = np.random.default_rng(H * d)
    qw, kw, eps = 1 + 0.4 * rng.standard_normal(d), 1 + 0.4 * rng.standard_normal(d), 1e-3
    for pos0, T in ((0, 9), (297, 5)):
        proj = rng.standard_normal((T, H * d + G * d + G * dv))
        proj[:, :d] *= 20.0
        q, k = proj[:, :H * d].reshape(T, H, d), proj[:, H * d:(H + G) * d].reshape(T, G, d)
        temp = np.array([O.query_temperature(pos0 + t, {"coef": coef, "every": every} if every else None) for t in range(T)])
        gq, kc, vc = capi.head_norm_post(proj, pos0, H, G, d, dv, qw, kw, eps, every, coef)
        close(gq, (O.rms_norm(q, qw, eps) * temp[:, None, None]).reshape(T, -1), F32_TOL)
        close(kc[pos0:], O.rms_norm(k, kw, eps).reshape(T, -1), F32_TOL)
        close(vc[pos0:], proj[:, (H + G) * d:], 1e-6)


def attention_reference(q, k, v, pos0, scale, slopes, gate=None):
    o = O.biased_attention(q, k, v, pos0, scale, slopes)
    if gate is not None:
        o = o / (1.0 + np.exp(-gate))[:, :, None]
    return o.reshape(q.shape[0], -1)


@pytest.mark.parametrize("H,G,d,dv", [(4, 1, 8, 8), (2, 2, 5, 3), (6, 3, 16, 24), (8, 2, 64, 64), (1, 1, 130, 7), (5, 1, 12, 20)])
@pytest.mark.parametrize("T,pos0,splits", [(1, 0, 1), (1, 300, 1), (1, 300, 5), (3, 97, 1), (40, 0, 1), (37, 60, 2)])
def test_distance_biased_attention(H, G, d, dv, T, pos0, splits):
    """Slopes 2^(-8(h+1)/H), the extra one in the denominator, a gate per head: one, a few and many queries take different kernels; key splits
    join partial sums before the extra one is added."""
    rng = np.random.default_rng(H * d + T + pos0)
    n = pos0 + T
    q, k, v, gate = rng.standard_normal((T, H, d)), rng.standard_normal((n, G, d)), rng.standard_normal((n, G, dv)), 2 * rng.standard_normal((T, H))
    slopes = O.head_slopes(H)
    f = lambda a: a.reshape(a.shape[0], -1)
    kw = dict(slope=slopes, sink=np.zeros(H), n_splits=splits)
    close(capi.biased_attention(f(q), f(k), f(v), pos0, H, G, d, dv, 0.4, gate=gate, **kw), attention_reference(q, k, v, pos0, 0.4, slopes, gate), F32_TOL)
    close(capi.biased_attention(f(q), f(k), f(v), pos0, H, G, d, dv, 0.4, **kw), attention_reference(q, k, v, pos0, 0.4, slopes), F32_TOL)
    close(capi.biased_attention(f(q), f(k), f(v), pos0, H, G, d, dv, 0.4, gate=gate, cache_bf16=True, **kw),
          attention_reference(q, O.bf16_round(k), O.bf16_round(v), pos0, 0.4, slopes, gate), F32_TOL)


def test_many_wide_heads_over_one_key_head():
    """So many that the launcher runs the heads in several launches: slopes, sinks and gates must follow their heads."""
    rng = np.random.default_rng(5)
    H, d, T, pos0 = 74, 256, 6, 40
    q, k, v, gate = rng.standard_normal((T, H, d)), rng.standard_normal((46, 1, d)), rng.standard_normal((46, 1, d)), rng.standard_normal((T, H))
    f = lambda a: a.reshape(a.shape[0], -1)
    got = capi.biased_attention(f(q), f(k), f(v), pos0, H, 1, d, d, 0.05, slope=O.head_slopes(H), sink=np.zeros(H), gate=gate)
    close(got, attention_reference(q, k, v, pos0, 0.05, O.head_slopes(H), gate), F32_TOL)


def test_the_extra_one_of_the_denominator_shows():
    """Scores far below zero: nearly all weight goes to the key that is not there; far above zero: none."""
    q, v = np.ones((1, 1, 4)), np.ones((3, 1, 2))
    for s, share in ((-9.0, 3 * math.exp(-9.0) / (1 + 3 * math.exp(-9.0))), (60.0, 1.0), (-80.0, 0.0)):
        got = capi.biased_attention(q.reshape(1, -1), np.full((3, 4), s / 4.0), v.reshape(3, -1), 2, 1, 1, 4, 2, 1.0, slope=[0.0], sink=[0.0])
        assert np.allclose(got, share, rtol=1e-5, atol=1e-12)


@pytest.mark.parametrize("far", [0, 1, 31, 32, 33, 255, 256, 700])
@pytest.mark.parametrize("T", [1, 3, 40])
def test_one_far_key_among_hundreds(far, T):
    """One query and one key are scaled so that their score stands out by more than the bias takes off over the whole distance: the output is
    that key's value, wherever the key lies.  The same score under a steep slope is lost: the bias is really the distance's."""
    rng = np.random.default_rng(far + T)
    H, G, d, n = 2, 1, 16, 760
    pos0 = n - T
    q, k, v = rng.standard_normal((T, H, d)), rng.standard_normal((n, G, d)), rng.standard_normal((n, G, d))
    k[far, 0] = 0.0
    k[far, 0, 3] = 10.0
    q[-1] = 0.0
    q[-1, :, 3] = 10.0
    slopes = [1.0, 2.0 ** -6]
    f = lambda a: a.reshape(a.shape[0], -1)
    got = capi.biased_attention(f(q), f(k), f(v), pos0, H, G, d, d, 0.45, slope=slopes, sink=np.zeros(H), n_splits=4 if T == 1 else 1)
    close(got[-1, d:], v[far, 0], 1e-4)
    want = attention_reference(q, k, v, pos0, 0.45, slopes)
    close(got, want, F32_TOL)
    if far < 700:
        assert np.abs(want[-1, :d] - v[far, 0]).max() > 0.1


def mixture_reference(x, h, w, top, E, correction, base, scale, other, other_scale):
    idx, wgt = O.route(h @ w["router"].T, correction, top)
    y = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, p in zip(idx[t], wgt[t]):
            y[t] += p * (O.gated_ff(h[t], w, f"e{e}.") if e < E else h[t])
    return x + scale * (y + base) + other_scale * other, idx, wgt


@pytest.mark.parametrize("K,ff,E,identity,top", [(12, 5, 4, 2, 3), (64, 16, 3, 1, 1), (40, 7, 5, 0, 5), (130, 33, 2, 6, 4), (512, 24, 33, 3, 8)])
@pytest.mark.parametrize("T", [1, 3, 50])
def test_mixture_with_identity_experts(K, ff, E, identity, top, T):
    """A correction larger than the scores decides most choices while the weights stay the scores; identity experts return the row itself; base,
    scale and the second sublayer's row join in one kernel.  Few pairs run as matvecs, many as sorted tiles."""
    rng = np.random.default_rng(K + T + top)
    w = {"router": rng.standard_normal((E + identity, K)) / math.sqrt(K) * 2}
    for e in range(E):
        w[f"e{e}.gate"], w[f"e{e}.up"] = rng.standard_normal((ff, K)) / math.sqrt(K), rng.standard_normal((ff, K)) / math.sqrt(K)
        w[f"e{e}.down"] = rng.standard_normal((K, ff)) / math.sqrt(ff)
    h, x, base, other = (rng.standard_normal((T, K)) for _ in range(4))
    scale, other_scale, corr = rng.standard_normal(K), rng.standard_normal(K), rng.standard_normal(E + identity)
    want, idx, wgt = mixture_reference(x, h, w, top, E, corr, base, scale, other, other_scale)
    stack = lambda leaf: np.stack([w[f"e{e}.{leaf}"] for e in range(E)])
    args = (w["router"], stack("gate"), stack("up"), stack("down"), top)
    got, gi, gw = capi.moe_join(x, h, *args, correction=corr, base=base, scale=scale, other=other, other_scale=other_scale)
    assert np.array_equal(gi, idx)
    close(gw, wgt, 1e-5)
    close(got, want, F32_TOL)
    if top < E + identity:
        assert not np.array_equal(np.sort(idx), np.sort(O.route(h @ w["router"].T, 0 * corr, top)[0]))   # the correction does decide something
    plain, pi, _ = mixture_reference(x, h, w, top, E, 0 * corr, 0.0, 1.0, 0.0, 0.0)
    got, gi, _ = capi.moe_join(x, h, *args)
    assert np.array_equal(gi, pi)
    close(got, plain, F32_TOL)


@pytest.mark.parametrize("T", [2, 40])
def test_only_identity_experts_chosen(T):
    rng = np.random.default_rng(T)
    E, K, ff = 3, 8, 4
    h, x, router = rng.standard_normal((T, K)), rng.standard_normal((T, K)), rng.standard_normal((E + 2, K))
    z = rng.standard_normal((E, ff, K))
    got, idx, wgt = capi.moe_join(x, h, router, z, z, rng.standard_normal((E, K, ff)), 2, correction=[0, 0, 0, 5.0, 9.0])
    assert (idx == [4, 3]).all()
    s = np.exp(h @ router.T)
    s /= s.sum(-1, keepdims=True)
    close(wgt, s[:, [4, 3]], 1e-5)
    close(got, x + (s[:, 4] + s[:, 3])[:, None] * h, F32_TOL)


def test_row_product_with_an_addend():
    rng = np.random.default_rng(8)
    for T, N, K in ((1, 7, 4), (3, 66, 16), (9, 33, 3), (70, 130, 8)):
        x, w, add = rng.standard_normal((T, K)), rng.standard_normal((N, K)), rng.standard_normal((T, N))
        close(capi.rows_add(x, w, add), x @ w.T + add, F32_TOL)


# ---- whole models ----------------------------------------------------------------------------------------------------------
A, M = O.attention_layer, O.moe
CONFIGS = {
    # a loop over the middle layers, unequal head sizes, a layer without a mixture, mixtures with and without identity / shared experts
    "mixed": O.make_config(vocab=41, width=24, mult=0.7, loop=(1, 3, 2), layers=[
        A(4, 2, 6, 5, 0.4, (0.5, 16), mlp=M(7, 5, 2, identity=2, shared=9)),
        A(6, 1, 8, 10, 0.35, (0.9, 3), mlp=M(6, 3, 3)),
        A(3, 3, 4, 4, 0.5, None, mlp=None),
        A(2, 1, 10, 3, 0.3, (0.3, 50), mlp=M(4, 2, 2, identity=3))]),
    # sizes of one: one head, one expert, width-one steps of the temperature, no loop
    "ones": O.make_config(vocab=17, width=16, mult=1.0, layers=[
        A(1, 1, 5, 7, 0.4, (0.2, 1), mlp=M(1, 1, 1, shared=1)),
        A(2, 2, 1, 1, 1.0, None, mlp=M(3, 1, 1, identity=1))]),
    # the whole model is one loop run four times; head sizes above a warp
    "loop_all": O.make_config(vocab=29, width=40, mult=0.4, loop=(0, 2, 4), layers=[
        A(6, 3, 40, 36, 0.15, (0.7, 20), mlp=M(10, 9, 4, identity=1, shared=12)),
        A(5, 1, 33, 12, 0.2, (0.4, 10), mlp=M(5, 4, 4, identity=4, shared=3))]),
    # one pass over a loop at the end: it still begins with the product
    "loop_once": O.make_config(vocab=23, width=20, loop=(1, 2, 1), layers=[
        A(4, 4, 6, 6, 0.4, (0.5, 8), mlp=M(6, 4, 2, identity=1)),
        A(4, 2, 6, 6, 0.4, (0.5, 8), mlp=M(6, 4, 2, identity=1, shared=5))]),
    # shapes the tensor-core GEMM takes (K multiples of 64)
    "k64_tiles": O.make_config(vocab=64, width=128, mult=0.6, loop=(0, 1, 2), layers=[
        A(8, 2, 16, 24, 0.25, (0.5, 30), mlp=M(64, 6, 3, identity=2, shared=192)),
        A(4, 1, 32, 16, 0.2, None, mlp=M(128, 4, 2, shared=64))]),
}


@pytest.fixture(scope="module", params=sorted(CONFIGS))
def case(request):
    cfg = CONFIGS[request.param]
    W = O.random_weights(cfg, seed=len(request.param))
    tokens = np.random.default_rng(11).integers(0, cfg["vocab"], 75).tolist()
    layers = []
    logits = O.forward(cfg, W, tokens, {}, layers)
    return cfg, W, tokens, logits, layers


def on_gpu(cfg, W, precision, chunk=None, max_tokens=256):
    if chunk:
        capi.tune("seq_chunk", chunk)
    try:
        return Model.from_json(cfg, W, "F32" if precision == capi.PRECISION_F32 else "BF16").cuda(max_tokens=max_tokens, precision=precision)
    finally:
        capi.tune("seq_chunk", 256)


def step_all(m, tokens, cuts):
    """Feed `tokens` in portions of the given sizes (the last size repeats), every position's logits."""
    rows, p, i = [], 0, 0
    while p < len(tokens):
        n = min(cuts[min(i, len(cuts) - 1)], len(tokens) - p)
        rows.append(m.prefill(tokens[p:p + n], p, 2).reshape(n, -1))
        p += n
        i += 1
    return np.concatenate(rows)


@pytest.mark.parametrize("precision", [capi.PRECISION_F32, capi.PRECISION_BF16])
def test_prompt_in_one_pass_and_layer_runs(case, precision, monkeypatch):
    cfg, W, tokens, logits, layers = case
    monkeypatch.setenv("XALM_SEQ_KEEP_LAYERS", "1")
    m = on_gpu(cfg, W, precision)
    got = m.prefill(tokens, 0, 2)
    assert m.info("n_layers") == len(O.layer_runs(cfg)) == len(layers)
    for r in range(len(layers)):             # the first run that differs names the mechanism
        x = m.read_state(100 + r, len(tokens) * cfg["width"]).reshape(len(tokens), -1)
        if precision == capi.PRECISION_F32:
            close(x, layers[r], F32_TOL)
        else:
            rows_within(x, layers[r], BF16_TOL)
    if precision == capi.PRECISION_F32:
        close(got, logits, F32_TOL)
    else:
        rows_within(got, logits, BF16_TOL)
    m.close()


@pytest.mark.parametrize("chunk", [8, 16, 256])
@pytest.mark.parametrize("cuts", [[1], [2], [3, 2, 7, 1, 30], [40, 1], [75]])
def test_portions_and_token_by_token(case, chunk, cuts):
    """However the prompt is cut — into steps by the caller, into passes by the engine (chunk) — every position's logits agree with the
    oracle: prefill against token-by-token decoding, portions down to two tokens, cache rows of every run handed from pass to pass."""
    cfg, W, tokens, logits, _ = case
    m = on_gpu(cfg, W, capi.PRECISION_F32, chunk=chunk)
    close(step_all(m, tokens, cuts), logits, F32_TOL)
    m.close()


def test_side_branch_off_gives_the_same_rows(case):
    """Attention beside the mixture on two streams or one after the other on one: the same kernels, the same bits."""
    cfg, W, tokens, _, _ = case
    rows = []
    for overlap in (1, 0):
        capi.tune("seq_overlap", overlap)
        try:
            m = on_gpu(cfg, W, capi.PRECISION_F32, chunk=16)
            rows.append(step_all(m, tokens, [20, 1, 1, 9]))
            m.close()
        finally:
            capi.tune("seq_overlap", 1)
    assert np.array_equal(rows[0], rows[1])


def test_tensor_core_passes_match_the_fp32_kernels():
    cfg = CONFIGS["k64_tiles"]
    W = O.random_weights(cfg, seed=9)
    tokens = np.random.default_rng(4).integers(0, cfg["vocab"], 130).tolist()
    logits = O.forward(cfg, W, tokens, {})
    launches, outputs = {}, {}
    for tc in (1, 2, 0):
        capi.tune("seq_tc", tc)
        try:
            m = on_gpu(cfg, W, capi.PRECISION_BF16, chunk=64)
        finally:
            capi.tune("seq_tc", 1)
        got = []
        for cuts in ([130], [40, 33, 5, 18, 34]):        # passes of 32 tokens or more take the tensor cores, shorter ones the fp32 kernels
            outputs[tc] = step_all(m, tokens, cuts)
            rows_within(outputs[tc], logits, BF16_TOL)
            got.append(m.last_launch_count())
            m.release()
        m.close()
        launches[tc] = got
    assert launches[1] != launches[0]                    # the tensor-core path really ran (pack + GEMM + epilogue)
    rows_within(outputs[2], outputs[0], BF16_TOL / 4)    # hi + lo operand planes: the fp32 kernels' numbers but for rounding
    rows_within(outputs[1], outputs[0], BF16_TOL)


@pytest.mark.parametrize("E,top,identity,ff", [(2, 2, 1, 192), (7, 3, 0, 64), (40, 8, 4, 64), (1, 1, 3, 320)])
def test_experts_of_long_passes_share_one_grouped_product(E, top, identity, ff):
    """Few experts with several row tiles each (the last one partly filled), many experts with a handful of rows, matrices of more than one
    column tile, passes in which most pairs are identity experts: against the oracle, and the two-plane operands against the fp32 tiles."""
    cfg = O.make_config(vocab=50, width=128, max_positions=512, mult=0.5, layers=[A(2, 1, 16, 16, 0.25, None, mlp=M(ff, E, top, identity=identity))])
    W = O.random_weights(cfg, seed=E)
    if E == 1:
        W["l0.mlp.correction"] = np.array([0.0, 0.6, 0.0, 0.0])
    tokens = np.random.default_rng(E).integers(0, 50, 410).tolist()
    logits = O.forward(cfg, W, tokens, {})
    out = {}
    for tc, moe_tc in ((1, 1), (2, 1), (2, 0)):
        capi.tune("seq_tc", tc)
        capi.tune("seq_moe_tc", moe_tc)
        try:
            m = on_gpu(cfg, W, capi.PRECISION_BF16, chunk=512, max_tokens=512)
        finally:
            capi.tune("seq_tc", 1)
            capi.tune("seq_moe_tc", 1)
        out[tc, moe_tc] = step_all(m, tokens, [410])
        rows_within(out[tc, moe_tc], logits, BF16_TOL)
        m.release()
        rows_within(step_all(m, tokens, [150, 33, 227]), logits, BF16_TOL)
        m.close()
    close(out[2, 1], out[2, 0], 1e-3)
    rows_within(out[1, 1], out[2, 0], BF16_TOL / 4)


def test_forward_steps_use_the_graph_and_match(case):
    cfg, W, tokens, logits, _ = case
    m = on_gpu(cfg, W, capi.PRECISION_F32, chunk=16)
    state = InferenceState(m.config)
    m.prefill(tokens[:30], 0, 0)
    for p in range(30, len(tokens)):
        m.forward(state, tokens[p], p)
        close(state.logits(), logits[p], F32_TOL)
    with pytest.raises(capi.XalmError):        # a step must continue where the sequence stands
        m.forward(state, 1, 3)
    m.close()


def test_released_rows_are_used_again(case):
    cfg, W, tokens, logits, _ = case
    m = on_gpu(cfg, W, capi.PRECISION_F32, chunk=8)
    other = [(t * 7 + 3) % cfg["vocab"] for t in tokens]
    for n in (75, 50, 3):                      # a longer, a shorter and a very short sequence leave their rows behind
        step_all(m, other[:n], [13])
        m.release()
        close(step_all(m, tokens, [20, 1, 1, 9]), logits, F32_TOL)
        m.release()
    m.close()


def test_requests_of_unequal_length_one_after_the_other(case):
    """Each request of a queue gives what it gives alone, whatever came before it."""
    cfg, W, tokens, _, _ = case
    m = on_gpu(cfg, W, capi.PRECISION_F32, chunk=16)
    for n, cuts in ((1, [1]), (60, [60]), (2, [2]), (33, [32, 1]), (17, [2, 3])):
        seq = [(t + n) % cfg["vocab"] for t in tokens[:n]]
        close(step_all(m, seq, cuts), O.forward(cfg, W, seq, {}), F32_TOL)
        m.release()
    m.close()


@pytest.mark.parametrize("precision,tol", [(capi.PRECISION_F32, 2 * F32_TOL), (capi.PRECISION_BF16, BF16_TOL)])
def test_long_decoding_to_the_last_position(precision, tol):
    """196 single steps up to the end of the position table, which also bounds a cache that was asked to be larger."""
    cfg = dict(CONFIGS["mixed"], max_positions=200)
    W = O.random_weights(cfg, seed=5)
    tokens = np.random.default_rng(2).integers(0, cfg["vocab"], 200).tolist()
    logits = O.forward(cfg, W, tokens, {})
    m = on_gpu(cfg, W, precision, chunk=8, max_tokens=1000)
    assert m.info("max_tokens") == 200
    got = step_all(m, tokens, [4, 1])
    if precision == capi.PRECISION_F32:
        close(got, logits, tol)
    else:
        rows_within(got, logits, tol)
    with pytest.raises(capi.XalmError, match="max_tokens"):
        m.prefill(tokens[:1], 200, 1)
    m.close()


def test_first_tokens_and_tiny_sequences(case):
    cfg, W, tokens, logits, _ = case
    m = on_gpu(cfg, W, capi.PRECISION_F32)
    for n in (1, 2, 3):
        close(m.prefill(tokens[:n], 0, 2), logits[:n], F32_TOL)
        m.release()
    m.close()


def far_config():
    cfg = O.make_config(vocab=31, width=32, max_positions=640, mult=1.0, loop=(0, 1, 2), layers=[A(1, 1, 16, 16, 1.0, (0.5, 64), mlp=None)])
    W = O.random_weights(cfg, seed=3)
    W["pos"] *= 0.0625                         # tokens, not positions, decide what a key says
    W["l0.norm1.b"] *= 0.0
    for n in ("l0.mix.q.norm", "l0.mix.k.norm"):
        W[n] = O.bf16_round(np.full(16, 1.5))
    W["l0.mix.k"] = -W["l0.mix.q"]             # a query scores highest with the key of the opposite row, lowest with its own
    W["embed"][29] = -W["embed"][30]
    return cfg, W


def test_a_far_token_decides_the_answer():
    """The last token's opposite occurs once, at position 15: that key's score stands above every other, so that the logits depend on a value
    hundreds of positions back, in a prompt and when decoding, across pass borders (chunk 64) and key blocks."""
    cfg, W = far_config()
    tokens = np.random.default_rng(6).integers(0, 29, 600).tolist()
    tokens[15], tokens[-1] = 29, 30
    logits = O.forward(cfg, W, tokens, {})
    other = list(tokens)
    other[15] = 7
    assert np.abs(O.forward(cfg, W, other, {})[-1] - logits[-1]).max() > 1.0        # position 15 decides the logits at position 599
    m = on_gpu(cfg, W, capi.PRECISION_F32, chunk=64, max_tokens=640)
    for cuts in ([600], [570, 1], [64, 65, 2]):
        close(step_all(m, tokens, cuts), logits, 2 * F32_TOL)
        m.release()
    m.close()


def test_greedy_generation_through_the_host_entry_points(case, tmp_path):
    cfg, W, tokens, _, _ = case
    prompt, steps = tokens[:12], 10
    seq = list(prompt)                         # the oracle generates greedily, recomputing the whole sequence each step
    for _ in range(steps):
        seq.append(int(np.argmax(O.forward(cfg, W, seq, {})[-1])))
    m = on_gpu(cfg, W, capi.PRECISION_F32, chunk=8)
    state, sampler = InferenceState(m.config), Sampler(m.config)
    assert generate(m, state, sampler, prompt, steps) == seq
    m.release()
    assert generate(m, state, sampler, prompt, steps, portion=5) == seq
    m.close()
    # the same through the command line on a model folder
    ST.write_model_dir(str(tmp_path / "model"), cfg, W, "BF16")
    build.build_host()
    out = subprocess.run([build.MAIN, str(tmp_path / "model"), "-p", "f32", "-T", "64", "-n", str(steps), "-i", " ".join(map(str, prompt))],
                         capture_output=True, text=True, check=True).stdout
    ids = [int(x) for x in out.split("\n")[1].split()]
    assert ids == seq[len(prompt):]


def test_trace_mode_of_the_command_line(case, tmp_path):
    cfg, W, tokens, logits, _ = case
    ST.write_model_dir(str(tmp_path / "model"), cfg, W, "BF16")
    (tmp_path / "out").mkdir()
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": tokens[:30], "want": [0, 29]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": tokens[30:32], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": tokens[32:33], "want": [0]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": tokens[:5], "want": [4]}], "end": ["b"]}]
    runner = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "bin", "trace_run")
    r = subprocess.run([runner, "--model", str(tmp_path / "model"), "--dtype", "float32", "--out", str(tmp_path / "out"), "--max-tokens", "64"],
                       input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, check=True)
    assert [l for l in r.stdout.split("\n") if l.startswith("done")] == ["done 0", "done 1", "done 2", "done 3"]
    V = cfg["vocab"]
    close(np.fromfile(tmp_path / "out" / "0.f32", dtype=np.float32).reshape(2, V), logits[[0, 29]], F32_TOL)
    assert not (tmp_path / "out" / "1.f32").exists()
    close(np.fromfile(tmp_path / "out" / "2.f32", dtype=np.float32).reshape(1, V), logits[[32]], F32_TOL)
    close(np.fromfile(tmp_path / "out" / "3.f32", dtype=np.float32).reshape(1, V), logits[[4]], F32_TOL)


def test_missing_tensors_are_named():
    for name in ("l0.norm1.b", "l0.mlp.correction", "loop.in", "pos", "final.norm.b", "l3.ls2"):
        W = O.random_weights(CONFIGS["mixed"], 1)
        del W[name]
        with pytest.raises(capi.XalmError, match=name):
            Model.from_json(CONFIGS["mixed"], W).cuda()
    W = O.random_weights(CONFIGS["mixed"], 1)
    W["l0.mix.g"] = W["l0.mix.g"][:2]
    with pytest.raises(capi.XalmError, match="l0.mix.g"):
        Model.from_json(CONFIGS["mixed"], W).cuda()
