"""Dotivik on the GPU against the plain restatement: every kernel alone (the layer norm with one and two additions, taken apart
into the products around it, with a mean far from zero; products with two sources, with a gated second part, and with another
base than the stream; gelu gates through each of their products; attention of two maps a head with a key far back, at page
borders and just inside and outside a window made to carry a map's weight, under caps that bind and caps that do not; latent
attention with a gate a head and windows cut into pieces; the paged write of two vectors a head), every kind of layer alone in
a small model, the stream after every run of a layer, whole prompts against portions, single tokens and mixed batches in pools
so small that pages are used again, long decoding, and greedy generation through the entry point and the command line."""

from types import SimpleNamespace

import numpy as np
import pytest
import torch

from tests import dotivik_util as U
from tests import replay_util as R
from tests.plain import dotivik_plain as P
from tests.test_gavodra_gpu import dev, fill_pools, hand_step, host, position_error, requests_for
from tests.test_rumedra_gpu import Limits, jittered_bfloat16, to_bfloat16

pytestmark = pytest.mark.gpu

# A position's error and its limits are those of the Rumedra tests: float32 a fixed part of the logits' spread, bfloat16
# three times what rounding does at that position in the plain restatement, and no less than FLOOR.
FLOOR = 0.03
BF16 = torch.bfloat16
GELU = dict(slope=2.0 * np.sqrt(2.0 / np.pi), cubic=0.044715)


def plain_logits(model_dir, reqs, dtype="float32"):
    cfg, w = U.read_config(model_dir), U.plain_weights(model_dir)
    out = Limits({name: P.forward(cfg, w, toks)[0] for name, toks in reqs.items()})
    out.limit = {}
    if dtype == "bfloat16":
        for name, toks in reqs.items():
            e = np.zeros(len(toks))
            for fn in (to_bfloat16, jittered_bfloat16(1)):
                with P.coarse_products(fn):
                    rounded = P.forward(cfg, w, toks)[0]
                e = np.maximum(e, [position_error(rounded[i], out[name][i]) for i in range(len(toks))])
            for i, x in enumerate(np.maximum(np.maximum(e, np.median(e)) * 3.0, FLOOR)):
                out.limit[(name, i)] = float(x)
    return out


def session(model_dir, dtype, max_tokens, page=16, max_live=4):
    from rust_llm_inference_server_b200.engine.replay import ReplaySession
    return ReplaySession(model_dir, dtype, max_tokens, page, max_live=max_live)


# ---- the kernels, one by one -------------------------------------------------------------------


@pytest.mark.parametrize("dtype", [torch.float32, BF16])
@pytest.mark.parametrize("T,W", [(3, 40), (7, 77), (1, 1030), (200, 192), (5, 2048), (70, 520)])
def test_layer_norm_with_one_and_two_additions(dtype, T, W):
    from rust_llm_inference_server_b200 import ops
    rng = np.random.default_rng(T * W)
    w, eps = 1 + 0.3 * rng.standard_normal(W), 1e-3
    tol = dict(rtol=0, atol=3e-5) if dtype == torch.float32 else dict(rtol=1e-2, atol=0.02)
    for mean in (0.0, 40.0):                               # a mean far from zero costs no digits
        x = rng.standard_normal((T, W)) + mean
        deltas = [host(dev(rng.standard_normal((T, W)), dtype)) for _ in range(2)]
        for n in (0, 1, 2):
            want_x = x + sum(deltas[:n]) if n else x
            want = P.layer_norm(want_x, w, eps)
            given = None if n == 0 else dev(deltas[0], dtype) if n == 1 else tuple(dev(d, dtype) for d in deltas)
            out, resid = torch.empty((T, W), dtype=dtype, device="cuda"), dev(x)
            rows = rng.integers(0, T, size=4)
            out4 = torch.empty((4, W), dtype=dtype, device="cuda")
            ops.layer_norm(resid, dev(w), eps, out4, given, dev(rows, torch.int32))
            assert torch.equal(resid, dev(x))              # rows only: the stream stays
            np.testing.assert_allclose(host(out4), want[rows], **tol)
            ops.layer_norm(resid, dev(w), eps, out, given)
            np.testing.assert_allclose(host(out), want, **tol)
            np.testing.assert_allclose(host(resid), want_x, rtol=0, atol=2e-5)
            resid = dev(x)
            ops.rmsnorm(resid, dev(w), eps, out, given)     # the RMS norm takes two additions as well
            np.testing.assert_allclose(host(out), P.rms_norm(want_x, w, eps), **tol)


@pytest.mark.parametrize("M,W,N,I,K,K2", [(1, 96, 40, 24, 64, 40), (8, 320, 104, 128, 512, 96), (16, 192, 8, 56, 72, 384),
                                          (5, 2048, 1000, 1024, 2048, 1504), (3, 1024, 3000, 64, 136, 8)])
def test_layer_norm_inside_the_products_around_it(M, W, N, I, K, K2):
    """A block of sublayers side by side: two products with one sum into the stream, the norm, and a stacked product whose
    second part is gated, against the operations one by one."""
    from rust_llm_inference_server_b200 import ops
    rng = np.random.default_rng(W + N)
    f = lambda *s: rng.standard_normal(s)
    x1, x2 = dev(f(M, K), BF16), dev(f(M, K2 + 16), BF16)[:, 8:8 + K2]            # the second a column slice
    w1, w2 = dev(f(W, K) / np.sqrt(K), BF16), dev(f(W, K2) / np.sqrt(K2), BF16)
    gain, eps = 1 + 0.3 * f(W), 1e-5
    w_in = dev(f(N + 2 * I, W) / np.sqrt(W), BF16)
    x, base = f(M, W) + 0.5, f(M, W) - 2.0
    y = host(x1) @ host(w1).T + host(x2) @ host(w2).T
    plain = host(w_in)
    gu = plain[N:].reshape(-1, 2, 4, W)
    np.testing.assert_allclose(host(ops.linear(x1, w1, second=(x2, w2))), y, rtol=1e-2, atol=0.03)
    for use_base in (False, True):
        resid = dev(x)
        sink = ops.ResidualSink(resid, dev(gain), eps, centred=True, base=dev(base) if use_base else None, exact=True)
        rows = ops.linear(x1, w1, sink=sink, second=(x2, w2))
        want_x = (base if use_base else x) + y
        np.testing.assert_allclose(host(resid), want_x, rtol=0, atol=3e-4)
        out, act = ops.stream_gemm(rows, w_in, n_plain=N, **GELU)
        h = P.layer_norm(want_x, gain, eps)
        want = h @ plain[:N].T
        want_act = P.gelu_tanh(h @ gu[:, 0].reshape(-1, W).T) * (h @ gu[:, 1].reshape(-1, W).T)
        assert out.shape == (M, N) and act.shape == (M, I)
        np.testing.assert_allclose(host(out), want, rtol=1e-2, atol=0.04)
        np.testing.assert_allclose(host(act), want_act, rtol=2e-2, atol=0.06)
        np.testing.assert_allclose(host(ops.linear(rows, w_in)), h @ plain.T, rtol=1e-2, atol=0.04)
        np.testing.assert_allclose(host(ops.linear(rows, w_in, out_dtype=torch.float32)), h @ plain.T, rtol=1e-2, atol=0.03)
    # rows that are normed already take the same stacked product
    hn = dev(h, BF16)
    out, act = ops.stream_gemm(hn, w_in, n_plain=N, **GELU)
    np.testing.assert_allclose(host(out), want, rtol=1e-2, atol=0.04)
    np.testing.assert_allclose(host(act), want_act, rtol=2e-2, atol=0.06)
    ops.check_device_errors()


def test_embedding_feeds_a_layer_norm_that_the_first_product_applies():
    from rust_llm_inference_server_b200 import ops
    rng = np.random.default_rng(2)
    for W in (40, 128, 1096):
        V, T, N = 33, 11, 72
        table, w = dev(rng.standard_normal((V, W)) + 1.0, BF16), dev(rng.standard_normal((N, W)) / np.sqrt(W), BF16)
        gain, ids = 1 + 0.3 * rng.standard_normal(W), rng.integers(0, V, size=T)
        out = torch.empty((T, W), device="cuda")
        rows = ops.embedding_sink(dev(ids, torch.int32), table, out, None, ops.ResidualSink(out, dev(gain), 1e-5, centred=True))
        assert torch.equal(out, table.float()[dev(ids, torch.long)])
        want = P.layer_norm(host(table)[ids], gain, 1e-5) @ host(w).T
        np.testing.assert_allclose(host(ops.linear(rows, w)), want, rtol=1e-2, atol=0.04)
        assert rows.weight is not None and ops.column_sums(w, rows.weight) is ops.column_sums(w, rows.weight)


@pytest.mark.parametrize("dtype", [torch.float32, BF16])
@pytest.mark.parametrize("T,W,I", [(3, 40, 24), (1, 128, 256), (16, 64, 100), (37, 100, 50), (150, 128, 256), (130, 64, 100), (300, 96, 384)])
def test_unit_gated_by_gelu(dtype, T, W, I):
    """Through its products for few rows, for a few dozen and for many (the gating in the product's epilogue where it can be)."""
    from rust_llm_inference_server_b200.parts.feed_forward import SwiGLU
    from rust_llm_inference_server_b200.parts.spec import GELU_TANH, SwiGLUSpec
    rng = np.random.default_rng(T + I)
    w = {n: dev(2 * rng.standard_normal(s) / np.sqrt(s[1]), dtype) for n, s in (("gate", (I, W)), ("up", (I, W)), ("down", (W, I)))}
    ff = SwiGLU(SwiGLUSpec(W, I, "gate", "up", "down", **GELU_TANH), dtype, "cuda")
    ff.load(SimpleNamespace(get=lambda name, role="matrix", share=False: w[name]))
    x = dev(rng.standard_normal((T, W)), dtype)
    st = SimpleNamespace(buffer=hand_step([1], [1], 8, 1, rng).buffer, n_tokens=T)
    plain = {k: host(v) for k, v in w.items()}
    with P.coarse_products(to_bfloat16 if dtype == BF16 else (lambda v: v)):
        want = P.gated_unit(host(x), plain, "")
    np.testing.assert_allclose(host(ff.forward(x, st)), want, rtol=0, atol=2e-4 if dtype == torch.float32 else 0.3)
    assert np.abs(P.linear(plain_silu(host(x), plain), plain["down"]) - want).max() > (0.1 if dtype == torch.float32 else 0.6)


def plain_silu(x, w):
    g = x @ w["gate"].T
    return g * P.sigmoid(g) * (x @ w["up"].T)


@pytest.mark.parametrize("dtype", [torch.float32, BF16])
@pytest.mark.parametrize("H,G,d,dv,dims,half", [(4, 2, 32, 16, 16, False), (3, 3, 24, 8, 24, False), (2, 1, 20, 12, 6, False),
                                                (6, 2, 64, 128, 32, True), (5, 1, 40, 72, 8, False), (2, 2, 10, 30, 4, True)])
def test_two_vectors_a_head_are_turned_and_stored_as_one_row(dtype, H, G, d, dv, dims, half):
    from rust_llm_inference_server_b200 import ops
    rng = np.random.default_rng(H * d)
    page, ctx, qn = 8, [40, 17, 1, 90], [5, 17, 1, 64]
    n_pages = 24
    st = hand_step(ctx, qn, page, n_pages, rng)
    T = st.n_tokens
    k_off, v_off = 2 * H * d, 2 * H * d + 2 * G * d
    N = -(-(v_off + G * dv + 5) // 8) * 8
    proj = dev(rng.standard_normal((T, N)), dtype)
    rot = {"dims": dims, "base": 77.0}
    freq = dev(77.0 ** (-2.0 * np.arange(dims // 2) / dims))
    x = host(proj)
    turn = P.rotate_halves if half else P.rotate_neighbours

    def turned(cols, heads):
        out = np.zeros((T, heads, d))
        for t in range(T):
            rows = np.zeros((st.host_pos[t] + 1, heads, d))
            rows[-1] = x[t, cols:cols + heads * d].reshape(heads, d)
            out[t] = turn(rows, rot)[-1]
        return out
    q_out = torch.empty((T, 2 * H * d), dtype=dtype, device="cuda")
    kc = torch.full((n_pages, G, page, 2 * d), 7.0, dtype=dtype, device="cuda")
    vc = torch.full((n_pages, G, page, dv), 7.0, dtype=dtype, device="cuda")
    ops.qk_norm_store(proj, 0, k_off, v_off, None, None, 1e-5, None, 0.0, q_out, kc, vc, st.slots[0], H, G, d, dv, page,
                      rotation=(freq, dims, 1.0), positions=st.positions, rot_half=half, maps=2)
    tol = dict(rtol=0, atol=2e-5) if dtype == torch.float32 else dict(rtol=1e-2, atol=0.01)
    np.testing.assert_allclose(host(q_out).reshape(T, 2 * H, d), turned(0, 2 * H), **tol)
    want_k = turned(k_off, 2 * G).reshape(T, G, 2 * d)
    touched = np.zeros((n_pages, page), dtype=bool)
    for t in range(T):
        pg, at = st.host_tables[st.host_seq[t], st.host_pos[t] // page], st.host_pos[t] % page
        touched[pg, at] = True
        np.testing.assert_allclose(host(kc[pg, :, at]), want_k[t], **tol)
        np.testing.assert_allclose(host(vc[pg, :, at]), x[t, v_off:v_off + G * dv].reshape(G, dv), rtol=0, atol=0)
    for c in (kc, vc):
        assert float((c.float().permute(0, 2, 1, 3)[~torch.from_numpy(touched).cuda()] - 7.0).abs().max()) == 0.0
