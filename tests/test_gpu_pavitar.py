"""Pavitar on the GPU against the plain restatement in tests/pavitar_oracle.py: every mechanism alone (op-level entry points that launch
the family's kernels), then whole models with small random configurations — prompts in one pass, token by token, in portions, after a
release, long decoding, keys on both sides of every window and chunk, greedy generation through the host entry points and the command line."""
import json
import math
import os
import subprocess

import numpy as np
import pytest

import pavitar_oracle as O
from xalm_b200 import build, capi
from xalm_b200 import safetensors_io as ST
from xalm_b200.model import InferenceState, Model, Sampler, generate

pytestmark = pytest.mark.gpu

F32_TOL = 2e-4   # IEEE fp32 path against float64, on values of order one
BF16_TOL = 6e-2  # serving mode: bf16 weights (exact here), bf16 caches, fp16 operands on the tensor cores


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


def flat(a):
    return a.reshape(a.shape[0], -1)


# ---- mechanisms alone ----------------------------------------------------------------------------------------------------
def frequencies(base, dims):
    return np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)])


@pytest.mark.parametrize("H,G,d,dv,dims", [(4, 2, 6, 9, 4), (1, 1, 1, 3, 0), (6, 3, 40, 8, 40), (8, 1, 128, 64, 64), (3, 1, 7, 5, 2), (16, 4, 128, 128, 96)])
@pytest.mark.parametrize("pos0,T", [(0, 9), (1300, 1), (797, 70)])
def test_row_norms_then_rotation(H, G, d, dv, dims, pos0, T):
    """One loud head pulls the whole row's norm; pairs of neighbours turn, the rest of a head passes; few and many tokens split their rows
    differently; an eps that matters; queries in place and apart; keys and values land in their ring slots."""
    rng = np.random.default_rng(H * d + T)
    eps, qw, kw = 0.3, 1 + 0.4 * rng.standard_normal(H * d), 1 + 0.4 * rng.standard_normal(G * d)
    proj = rng.standard_normal((T, H * d + G * d + G * dv))
    proj[:, :d] *= 20.0
    q = O.turn_pairs(O.rms_norm(proj[:, :H * d], qw, eps).reshape(T, H, d), pos0, 300.0, dims) if dims else O.rms_norm(proj[:, :H * d], qw, eps)
    k = O.rms_norm(proj[:, H * d:(H + G) * d], kw, eps)
    k = O.turn_pairs(k.reshape(T, G, d), pos0, 300.0, dims) if dims else k
    ring = T + 5
    for in_place in (False, True):
        gq, kc, vc = capi.row_norm_post(proj, pos0, H, G, d, dv, qw, kw, frequencies(300.0, dims) if dims else None, True, eps, ring, in_place)
        slots = (pos0 + np.arange(T)) % ring
        close(gq, flat(q), F32_TOL)
        close(kc[slots], flat(k), F32_TOL)
        close(vc[slots], proj[:, (H + G) * d:], 1e-6)
        assert np.abs(np.delete(kc, slots, 0)).max() == 0 and np.abs(np.delete(vc, slots, 0)).max() == 0


def test_row_norms_with_halves_turned():
    """The same kernel in the other layout of a head: entry i with i + half."""
    rng = np.random.default_rng(1)
    H, G, d, T, half = 3, 1, 10, 5, 3
    proj = rng.standard_normal((T, (H + G) * d + d))
    q = O.rms_norm(proj[:, :H * d], 1.0, 1e-5).reshape(T, H, d)
    a = (7 + np.arange(T))[:, None, None] * frequencies(50.0, 2 * half)
    want = q.copy()
    want[:, :, :half], want[:, :, half:2 * half] = q[:, :, :half] * np.cos(a) - q[:, :, half:2 * half] * np.sin(a), q[:, :, half:2 * half] * np.cos(a) + q[:, :, :half] * np.sin(a)
    close(capi.row_norm_post(proj, 7, H, G, d, d, None, None, frequencies(50.0, 2 * half), False)[0], flat(want), F32_TOL)


@pytest.mark.parametrize("H,G,d,dv", [(4, 1, 8, 8), (2, 2, 5, 3), (6, 3, 16, 24), (8, 2, 64, 64), (5, 1, 12, 20)])
@pytest.mark.parametrize("chunk", [1, 7, 32, 100])
@pytest.mark.parametrize("T,pos0,splits", [(1, 0, 1), (1, 299, 1), (1, 300, 5), (3, 97, 1), (3, 98, 2), (40, 0, 1), (37, 70, 2)])
def test_chunked_attention(H, G, d, dv, chunk, T, pos0, splits):
    """One, a few and many queries take different kernels; chunk borders fall inside query tiles and key blocks; a ring that holds no more than
    one chunk and the queries."""
    rng = np.random.default_rng(H * d + T + pos0 + chunk)
    n = pos0 + T
    q, k, v = rng.standard_normal((T, H, d)), rng.standard_normal((n, G, d)), rng.standard_normal((n, G, dv))
    sees = lambda i, j: O.sees_chunk(i, j, chunk)
    kw = dict(ring=min(n, chunk - 1 + T), n_splits=splits)
    close(capi.chunked_attention(flat(q), flat(k), flat(v), pos0, H, G, d, dv, chunk, 0.4, **kw), flat(O.attend(q, k, v, pos0, 0.4, sees)), F32_TOL)
    close(capi.chunked_attention(flat(q), flat(k), flat(v), pos0, H, G, d, dv, chunk, 0.4, cache_bf16=True, **kw),
          flat(O.attend(q, O.bf16_round(k), O.bf16_round(v), pos0, 0.4, sees)), F32_TOL)


@pytest.mark.parametrize("T", [1, 3, 40])
@pytest.mark.parametrize("i,chunk", [(255, 256), (256, 256), (500, 128), (639, 640), (97, 33), (98, 33), (99, 33)])
def test_a_key_on_either_side_of_a_chunk_border(i, chunk, T):
    """The key that stands out is the chunk's first (seen: the output is its value) or the one before it (not seen, however loud)."""
    rng = np.random.default_rng(i + T)
    H, G, d = 2, 1, 16
    pos0 = i + 1 - T
    first = i // chunk * chunk
    q, k, v = rng.standard_normal((T, H, d)), rng.standard_normal((i + 1, G, d)), rng.standard_normal((i + 1, G, d))
    q[-1] = 0.0
    q[-1, :, 3] = 10.0
    for loud, seen in ((first, True), (first - 1, False)):
        if loud < 0:
            continue
        kk = k.copy()
        kk[loud, 0] = 0.0
        kk[loud, 0, 3] = 10.0
        for splits in ((1, 4) if T == 1 else (1,)):
            got = capi.chunked_attention(flat(q), flat(kk), flat(v), pos0, H, G, d, d, chunk, 0.45, n_splits=splits)
            close(got, flat(O.attend(q, kk, v, pos0, 0.45, lambda a, b: O.sees_chunk(a, b, chunk))), F32_TOL)
            share = np.abs(got[-1, :d] - v[loud, 0]).max() < 1e-3
            assert share == (seen or bool(np.abs(v[loud, 0] - v[i, 0]).max() < 1e-3))


def latent_reference(q, c, uk, uv, pos0, scale, window, gate):
    T, H, d = q.shape
    k, v = (c @ uk.T).reshape(-1, H, d), (c @ uv.T).reshape(c.shape[0], H, -1)
    o = O.attend(q, k, v, pos0, scale, lambda i, j: O.sees_window(i, j, window))
    return flat(o if gate is None else o * O.sigmoid(gate)[:, :, None])


@pytest.mark.parametrize("H,d,dv,R", [(4, 8, 8, 24), (1, 1, 3, 1), (3, 5, 9, 40), (16, 32, 16, 64), (40, 16, 24, 256)])
@pytest.mark.parametrize("window", [1, 9, 64, 1000])
@pytest.mark.parametrize("T,pos0,splits", [(1, 0, 0), (1, 200, 0), (3, 97, 0), (40, 0, 0), (37, 70, 2)])
def test_latent_attention_in_a_window(H, d, dv, R, window, T, pos0, splits):
    """Expanded keys and values (oracle) against queries mapped into the latent (product), with and without a gate per head, a ring no larger than
    the window and the step; forty heads over a wide latent run in several launches, and the gates follow their heads."""
    rng = np.random.default_rng(H + R + T + window)
    n = pos0 + T
    q, c, gate = rng.standard_normal((T, H, d)), rng.standard_normal((n, R)), 2 * rng.standard_normal((T, H))
    uk, uv = rng.standard_normal((H * d, R)) / math.sqrt(R), rng.standard_normal((H * dv, R)) / math.sqrt(R)
    ring = min(n, window - 1 + T)
    for g in (gate, None):
        close(capi.latent_window(flat(q), c, pos0, H, d, dv, R, uk, uv, 0.5, window, g, ring, splits), latent_reference(q, c, uk, uv, pos0, 0.5, window, g), F32_TOL)
    close(capi.latent_window(flat(q), c, pos0, H, d, dv, R, uk, uv, 0.5, window, gate, ring, splits, cache_bf16=True),
          latent_reference(q, O.bf16_round(c), uk, uv, pos0, 0.5, window, gate), F32_TOL)


@pytest.mark.parametrize("T", [1, 3, 40])
@pytest.mark.parametrize("window", [2, 31, 32, 33, 100, 300])
def test_a_key_on_either_side_of_the_window(window, T):
    rng = np.random.default_rng(window + T)
    H, d, R, n = 2, 8, 16, 420
    pos0, i = n - T, n - 1
    q, c = rng.standard_normal((T, H, d)), 0.3 * rng.standard_normal((n, R))
    uk, uv = rng.standard_normal((H * d, R)), rng.standard_normal((H * d, R))
    u = np.eye(R)[5]
    for h in range(H):
        q[-1, h] = 8.0 * (uk[h * d:(h + 1) * d] @ u)
    for back, seen in ((window - 1, True), (window, False)):
        cc = c.copy()
        cc[i - back] = 4.0 * u
        got = capi.latent_window(flat(q), cc, pos0, H, d, d, R, uk, uv, 1.0, window, None, window - 1 + T)
        close(got, latent_reference(q, cc, uk, uv, pos0, 1.0, window, None), F32_TOL)
        assert (np.abs(got[-1] - 4.0 * (uv @ u)).max() < 1e-3) == seen


@pytest.mark.parametrize("K,ff,E,top", [(12, 5, 4, 3), (64, 16, 3, 1), (40, 7, 5, 5), (130, 33, 2, 2), (512, 24, 33, 8), (16, 4, 1, 1)])
@pytest.mark.parametrize("T", [1, 3, 50])
def test_mixture_weighted_among_the_chosen(K, ff, E, top, T):
    """The bias decides many choices and enters the weights; the shared row is gated per token; few pairs run as matvecs, many as sorted tiles."""
    rng = np.random.default_rng(K + T + top)
    w = {"router": rng.standard_normal((E, K)) / math.sqrt(K) * 2, "router.b": 1.5 * rng.standard_normal(E)}
    for e in range(E):
        w[f"e{e}.gate"], w[f"e{e}.up"] = rng.standard_normal((ff, K)) / math.sqrt(K), rng.standard_normal((ff, K)) / math.sqrt(K)
        w[f"e{e}.down"] = rng.standard_normal((K, ff)) / math.sqrt(ff)
    h, x, base = (rng.standard_normal((T, K)) for _ in range(3))
    sg = rng.standard_normal(K) / math.sqrt(K) * 3
    stack = lambda leaf: np.stack([w[f"e{e}.{leaf}"] for e in range(E)])
    args = (w["router"], stack("gate"), stack("up"), stack("down"), top)
    mlp = {"router": {"experts": E, "top": top}}
    got, gi, gw = capi.moe_chosen(x, h, *args, bias=w["router.b"], base=base, gate_row=sg)
    idx, wgt = O.route(h @ w["router"].T + w["router.b"], top)
    assert np.array_equal(gi, idx)
    close(gw, wgt, 1e-5)
    close(gw.sum(1), np.ones(T), 1e-5)
    close(got, x + O.expert_ff(h, mlp, w, "") + O.sigmoid(h @ sg)[:, None] * base, F32_TOL)
    close(capi.moe_chosen(x, h, *args, base=base)[0], x + O.expert_ff(h, mlp, dict(w, **{"router.b": np.zeros(E)}), "") + base, F32_TOL)


def test_weights_of_far_apart_logits():
    """Logits hundreds apart: a softmax over all experts would have no room left for the second choice's neighbours; the order is the logits'."""
    E, K = 6, 4
    h, router = np.ones((2, K)), np.zeros((E, K))
    bias = np.array([-400.0, -401.0, 300.0, -402.0, -399.5, 0.0])
    z = np.zeros((E, 2, K))
    _, idx, wgt = capi.moe_chosen(np.zeros((2, K)), h, router, z, z, np.zeros((E, K, 2)), 4, bias=bias)
    assert (idx == [2, 5, 4, 0]).all()
    close(wgt, np.tile([1.0, 0, 0, 0], (2, 1)), 1e-6)
    _, idx, wgt = capi.moe_chosen(np.zeros((2, K)), h, router, z, z, np.zeros((E, K, 2)), 2, bias=np.array([-400.0, -401.0, -900.0, -402.0, -399.5, -999.0]))
    assert (idx == [4, 0]).all()
    close(wgt, np.tile(np.array([1.0, math.exp(-0.5)]) / (1 + math.exp(-0.5)), (2, 1)), 1e-5)


# ---- whole models ----------------------------------------------------------------------------------------------------------
L, A, M = O.latent_layer, O.attention_layer, O.moe
CONFIGS = {
    # a loop over the middle layers, unequal head sizes, windows and chunks that divide nothing, with and without shared experts, a layer without mixture
    "mixed": O.make_config(vocab=41, width=24, loop=(1, 3, 3), layers=[
        L(4, 6, 5, 10, 14, 9, 0.5, mlp=M(7, 5, 2, shared=9)),
        A(6, 2, 8, 10, 13, 0.4, (100.0, 6), mlp=M(6, 3, 3)),
        L(3, 4, 7, 8, 20, 31, 0.6, mlp=None),
        A(3, 3, 4, 4, 40, 0.5, (1e4, 4), mlp=M(4, 6, 1, shared=11))]),
    # sizes of one: one head, one expert, a window and a chunk of one position, a latent of one, odd heads; no cap on the logits
    "ones": O.make_config(vocab=17, width=16, cap=None, layers=[
        L(1, 1, 3, 1, 1, 1, 1.0, mlp=M(1, 1, 1, shared=1)),
        A(1, 1, 5, 7, 1, 0.4, (10.0, 2), mlp=M(3, 2, 1)),
        L(5, 3, 1, 2, 3, 2, 0.7, mlp=M(2, 2, 2, shared=3)),
        A(2, 1, 3, 1, 2, 0.5, (10.0, 2), mlp=None)]),
    # the whole model is one loop run four times; head sizes above a warp, one key head
    "loop_all": O.make_config(vocab=29, width=40, cap=30.0, loop=(0, 2, 4), layers=[
        A(6, 1, 40, 36, 50, 0.2, (500.0, 24), mlp=M(10, 9, 4, shared=12)),
        L(5, 33, 12, 24, 48, 24, 0.2, mlp=M(5, 4, 4, shared=3))]),
    # one pass over a loop at the end: nothing is added; only latent layers; windows beyond the prompt
    "loop_once": O.make_config(vocab=23, width=20, loop=(1, 2, 1), layers=[
        L(4, 6, 6, 12, 16, 500, 0.4, mlp=M(6, 4, 2, shared=7)),
        L(2, 8, 3, 9, 11, 17, 0.4, mlp=M(6, 4, 2, shared=5))]),
    # shapes the tensor-core GEMM takes (K multiples of 64), loop at the end
    "k64_tiles": O.make_config(vocab=64, width=128, eps=1e-6, loop=(1, 2, 2), layers=[
        L(8, 16, 24, 64, 128, 33, 0.25, mlp=M(64, 6, 3, shared=192)),
        A(4, 2, 32, 16, 48, 0.2, (1e4, 16), mlp=M(128, 4, 2, shared=64))]),
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
    oracle: prefill against token-by-token decoding, portions down to two tokens, rings that wrap, rows of every run handed from pass to pass."""
    cfg, W, tokens, logits, _ = case
    m = on_gpu(cfg, W, capi.PRECISION_F32, chunk=chunk)
    close(step_all(m, tokens, cuts), logits, F32_TOL)
    m.close()


def test_tensor_core_passes_match_the_fp32_kernels():
    cfg = CONFIGS["k64_tiles"]
    W = O.random_weights(cfg, seed=9)
    tokens = np.random.default_rng(4).integers(0, cfg["vocab"], 130).tolist()
    logits = O.forward(cfg, W, tokens, {})
    launches, outputs = {}, {}
    for tc in (1, 2, 0):
        capi.tune("seq_tc", tc)
        try:
            m = on_gpu(cfg, W, capi.PRECISION_BF16)
            outputs[tc] = m.prefill(tokens, 0, 2)
            launches[tc] = m.last_launch_count()
            rows_within(outputs[tc], logits, BF16_TOL)
            m.close()
        finally:
            capi.tune("seq_tc", 1)
    assert launches[1] > launches[0]           # the tensor-core path really ran (its GEMMs pack their operands first)
    rows_within(outputs[2], outputs[0], 1e-2)


def test_side_branch_off_gives_the_same_rows(case):
    """The router beside the shared expert on two streams or before it on one: the same kernels, the same bits."""
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


def test_graph_and_eager_steps_agree(case):
    cfg, W, tokens, _, _ = case
    rows = []
    for graph in (1, 0):
        capi.tune("seq_graph", graph)
        try:
            m = on_gpu(cfg, W, capi.PRECISION_F32, chunk=16)
            rows.append(step_all(m, tokens, [20, 1]))
            m.close()
        finally:
            capi.tune("seq_graph", 1)
    assert np.array_equal(rows[0], rows[1])


def test_unequal_requests_one_after_another(case):
    """A queue of requests of different lengths through one handle: rings and pass buffers are used again after release, and every request gives
    what it gives alone — also when the one before left a longer past behind."""
    cfg, W, tokens, _, _ = case
    m = on_gpu(cfg, W, capi.PRECISION_F32, chunk=16, max_tokens=80)
    rng = np.random.default_rng(3)
    for n, cuts in ((75, [75]), (1, [1]), (33, [16, 1]), (2, [2]), (60, [30, 2]), (18, [1])):
        seq = tokens[:n] if n == 75 else rng.integers(0, cfg["vocab"], n).tolist()
        close(step_all(m, seq, cuts), O.forward(cfg, W, seq, {}), F32_TOL)
        with pytest.raises(capi.XalmError):
            m.prefill(seq[:1], n + 1, 1)       # not where the sequence stands
        m.release()
    m.close()


@pytest.mark.parametrize("precision,tol", [(capi.PRECISION_F32, 2 * F32_TOL), (capi.PRECISION_BF16, BF16_TOL)])
def test_long_decoding(precision, tol):
    """Three hundred single steps: every ring wraps many times, chunks end and begin while decoding."""
    cfg = CONFIGS["mixed"]
    W = O.random_weights(cfg, seed=5)
    tokens = np.random.default_rng(2).integers(0, cfg["vocab"], 304).tolist()
    logits = O.forward(cfg, W, tokens, {})
    m = on_gpu(cfg, W, precision, chunk=8, max_tokens=304)
    got = step_all(m, tokens, [4, 1])
    if precision == capi.PRECISION_F32:
        close(got, logits, tol)
    else:
        rows_within(got, logits, tol)
    with pytest.raises(capi.XalmError, match="max_tokens"):
        m.prefill(tokens[:1], 304, 1)
    m.close()


def test_first_tokens_and_tiny_sequences(case):
    cfg, W, tokens, logits, _ = case
    m = on_gpu(cfg, W, capi.PRECISION_F32)
    for n in (1, 2, 3):
        close(m.prefill(tokens[:n], 0, 2), logits[:n], F32_TOL)
        m.release()
    m.close()


def edge_model(kind, size):
    """One mixer, no mixture: a query scores far highest with the key of the opposite row (tokens 29 and 30 are opposites)."""
    layer = L(1, 16, 16, 24, 24, size, 1.0) if kind == "window" else A(1, 1, 16, 16, size, 1.0, (1e6, 2))
    cfg = O.make_config(vocab=31, width=32, cap=60.0, layers=[layer])
    W = O.random_weights(cfg, seed=3)
    W["embed"][29] = -W["embed"][30]
    if kind == "window":
        W["l0.mix.dkv"] = -W["l0.mix.dq"]
        W["l0.mix.uq"] = W["l0.mix.uk"]
        W["l0.mix.dq.norm"] = W["l0.mix.dkv.norm"] = np.full(24, 1.0)
        W["l0.mix.g"] = np.abs(W["l0.mix.g"]) * np.sign(W["embed"][30])     # token 30's gate is open
    else:
        W["l0.mix.k"] = -W["l0.mix.q"]
        W["l0.mix.q.norm"] = W["l0.mix.k.norm"] = np.full(16, 1.5)
    return cfg, W


@pytest.mark.parametrize("kind,size,n", [("window", 40, 150), ("window", 257, 600), ("window", 64, 65), ("chunk", 50, 150), ("chunk", 256, 500), ("chunk", 64, 128)])
def test_edges_of_windows_and_chunks_in_prompts_and_decoding(kind, size, n):
    """The last token's opposite stands at the last visible place (it decides the logits) or one before it (they are what they are without it);
    the prompt in one step, the last tokens one by one, and portions that end next to the edge."""
    cfg, W = edge_model(kind, size)
    edge = n - size if kind == "window" else (n - 1) // size * size
    base = np.random.default_rng(6).integers(0, 29, n).tolist()
    base[-1] = 30
    last = {}
    m = on_gpu(cfg, W, capi.PRECISION_F32, chunk=64, max_tokens=n)
    for place in (edge, edge - 1, None):
        tokens = list(base)
        if place is not None and place >= 0:
            tokens[place] = 29
        logits = O.forward(cfg, W, tokens, {})
        last[place] = logits[-1]
        for cuts in ([n], [n - 5, 1], [edge, 2, 64] if edge > 0 else [3, 64], [63, 65, 2]):
            close(step_all(m, tokens, cuts), logits, 2 * F32_TOL)
            m.release()
    m.close()
    assert np.abs(last[edge] - last[None]).max() > 0.5
    assert np.abs(last[edge - 1] - last[None]).max() < 1e-9


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
    for name in ("l0.norm2", "l0.mix.dq.norm", "l0.mix.g", "l1.mix.k.norm", "l0.mlp.router.b", "l3.mlp.shared.sg", "final.norm", "l1.mlp.e2.down"):
        W = O.random_weights(CONFIGS["mixed"], 1)
        del W[name]
        with pytest.raises(capi.XalmError, match=name):
            Model.from_json(CONFIGS["mixed"], W).cuda()
    W = O.random_weights(CONFIGS["mixed"], 1)
    W["l1.mix.q.norm"] = W["l1.mix.q.norm"][:8]
    with pytest.raises(capi.XalmError, match="l1.mix.q.norm"):
        Model.from_json(CONFIGS["mixed"], W).cuda()
