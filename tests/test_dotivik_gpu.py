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


DIFF_SHAPES = [(4, 2, 32, 16, 8), (3, 3, 24, 8, 16), (1, 1, 8, 24, 16), (6, 2, 64, 128, 16), (8, 1, 64, 64, 32), (16, 2, 48, 96, 64),
               (10, 1, 40, 72, 16), (2, 1, 72, 136, 16), (5, 5, 20, 12, 16), (2, 2, 56, 120, 8)]


def plain_difference_rows(q, keys, vals, scale, cap, window, lam, diff, eps, gate, st, H, G):
    T = q.shape[0]
    out = np.zeros((T, H, vals[0].shape[-1]))
    for t in range(T):
        b, pos = st.host_seq[t], st.host_pos[t]
        lo = max(0, pos - window + 1) if window else 0
        for h in range(H):
            g = h // (H // G)
            a = []
            for m in (0, 1):
                s = keys[b][lo:pos + 1, g, m] @ q[t, h, m] * scale
                a.append(P.softmax(P.capped(s, cap) if cap else s) @ vals[b][lo:pos + 1, g])
            out[t, h] = P.difference_of_maps(a[0], a[1], lam, diff, eps)
    return out * P.sigmoid(gate)[:, :, None]


@pytest.mark.parametrize("dtype", [torch.float32, BF16])
@pytest.mark.parametrize("cap,window", [(50.0, 0), (9.0, 0), (90.0, 0), (0.0, 0), (40.0, 70), (0.0, 33)])
@pytest.mark.parametrize("H,G,d,dv,page", DIFF_SHAPES)
def test_attention_of_two_maps_far_keys_page_borders_and_windows(dtype, H, G, d, dv, page, cap, window):
    """Whole prompts, portions that start in the middle of a page, and single tokens in one launch.  Per head and map one key
    is made to carry the weight (query and key scaled): the first token, a page's last and first slot, a key far back, the
    token itself, and with a window the keys just inside and just outside its edge."""
    from rust_llm_inference_server_b200 import ops
    rng = np.random.default_rng(H * 100 + d)
    ctx, qn = [150, 70, 129, 1, 2, 900, 65, 420], [150, 1, 37, 1, 2, 1, 64, 1]
    n_pages = sum(-(-c // page) for c in ctx) + 3
    st = hand_step(ctx, qn, page, n_pages, rng)
    T, scale, lam, diff, eps = st.n_tokens, 0.7 / np.sqrt(d), 0.62, 0.3, 1e-5
    keys, vals = [rng.standard_normal((c, G, 2, d)) for c in ctx], [rng.standard_normal((c, G, dv)) for c in ctx]
    q = rng.standard_normal((T, H, 2, d))
    for t in range(T):
        b, pos = st.host_seq[t], st.host_pos[t]
        spots = [0, (pos // page) * page - 1, (pos // page) * page, pos // 2, pos, pos - window + 1, pos - window, pos - 1]
        for h in range(H):
            for m in (0, 1):
                j = min(max(spots[(h + 3 * m + t) % len(spots)], 0), pos)
                k = keys[b][j, h // (H // G), m]
                q[t, h, m] = k * (11.0 / scale / float(k @ k)) if (t + h) % 3 else q[t, h, m]
    gate = dev(rng.standard_normal((T, H + 11)) * 2, dtype)[:, 8:8 + H]
    qd, out = dev(q.reshape(T, -1), dtype), torch.full((T, H * dv), float("nan"), dtype=dtype, device="cuda")
    kr = [host(dev(k.reshape(k.shape[0], G, 2 * d), dtype)) for k in keys]
    vr = [host(dev(v, dtype)) for v in vals]
    kc, vc = fill_pools(st, kr, vr, page, n_pages, dtype)
    ops.launches_by_kernel.clear()
    ops.attention_difference(qd, kc, vc, out, gate, st, 0, H, G, d, dv, page, scale, cap, lam, 1.0 - diff, eps, window)
    args = (host(qd).reshape(T, H, 2, d), [k.reshape(-1, G, 2, d) for k in kr], vr, scale)
    want, got = plain_difference_rows(*args, cap, window, lam, diff, eps, host(gate), st, H, G), host(out).reshape(T, H, dv)
    err = np.abs(got - want).max(axis=(1, 2))
    assert np.isfinite(got).all() and err.max() <= (5e-5 if dtype == torch.float32 else 0.06), \
        f"row {int(err.argmax())} (request {st.host_seq[int(err.argmax())]}, position {st.host_pos[int(err.argmax())]}): {err.max()}"
    if cap == 9.0 or window:                                # the test bites
        other = plain_difference_rows(*args, 0.0 if cap == 9.0 else cap, window + 1 if window else 0, lam, diff, eps, host(gate), st, H, G)
        assert np.abs(other - want).max() > 0.08             # (two heads with keys that stand out less than elsewhere: 0.09)
    ran = set(ops.launches_by_kernel)
    if dtype == BF16 and ops.difference_prefill_takes_mma(dtype, d, dv, page):
        assert "attention_difference.prefill.tcgen05" in ran
    if dtype == BF16 and ops.difference_decode_takes_mma(dtype, H, G, d, dv):
        assert "attention_difference.decode.mma" + (".cluster" if not window else "") in ran
    ops.check_device_errors()


def test_single_tokens_whose_contexts_are_not_cut():
    """Contexts so short, and requests so many, that decode attention takes one piece each."""
    from rust_llm_inference_server_b200 import ops
    rng = np.random.default_rng(4)
    H, G, d, dv, page = 8, 2, 64, 128, 16
    ctx = [1, 2, 15, 16, 17, 63, 64, 65, 127, 100]
    st = hand_step(ctx, [1] * len(ctx), page, 60, rng)
    T = st.n_tokens
    keys, vals = [rng.standard_normal((c, G, 2 * d)) for c in ctx], [rng.standard_normal((c, G, dv)) for c in ctx]
    q = dev(rng.standard_normal((T, H * 2 * d)) * 2, BF16)
    kr, vr = [host(dev(k, BF16)) for k in keys], [host(dev(v, BF16)) for v in vals]
    kc, vc = fill_pools(st, kr, vr, page, 60, BF16)
    out = torch.full((T, H * dv), float("nan"), dtype=BF16, device="cuda")
    ops.launches_by_kernel.clear()
    ops.attention_difference(q, kc, vc, out, None, st, 0, H, G, d, dv, page, 0.2, 30.0, 0.5, 0.7, 1e-5)
    want = plain_difference_rows(host(q).reshape(T, H, 2, d), [k.reshape(-1, G, 2, d) for k in kr], vr, 0.2, 30.0, 0, 0.5, 0.3, 1e-5,
                                 np.full((T, H), 60.0), st, H, G)
    np.testing.assert_allclose(host(out).reshape(T, H, dv), want, rtol=0, atol=0.05)
    assert ops.launches_by_kernel == {"attention_difference.decode.mma": 1}


@pytest.mark.parametrize("dtype", [torch.float32, BF16])
@pytest.mark.parametrize("H,rank,rot,window,page", [(3, 40, 8, 7, 8), (6, 64, 32, 100, 16), (18, 128, 16, 600, 16), (2, 512, 64, 0, 32),
                                                    (1, 16, 2, 1, 16), (5, 256, 32, 64, 64)])
def test_latent_attention_with_a_gate_at_window_edges(dtype, H, rank, rot, window, page):
    from rust_llm_inference_server_b200 import ops
    rng = np.random.default_rng(rank + window)
    dk = rank + rot
    ctx, qn = [150, 70, 129, 1, 2, 1500, 65, 720], [150, 1, 37, 1, 2, 1, 64, 1]
    n_pages = sum(-(-c // page) for c in ctx) + 3
    st = hand_step(ctx, qn, page, n_pages, rng)
    T, scale = st.n_tokens, 0.5 / np.sqrt(dk)
    rows = [host(dev(rng.standard_normal((c, dk)), dtype)) for c in ctx]
    qa = rng.standard_normal((T, H, dk))
    for t in range(T):
        b, pos = st.host_seq[t], st.host_pos[t]
        spots = [pos - window + 1, pos - window, 0, (pos // page) * page, (pos // page) * page - 1, pos]
        for h in range(H):
            j = min(max(spots[(h + t) % len(spots)], 0), pos)
            if (t + h) % 3:
                qa[t, h] = rows[b][j] * (7.0 / scale / float(rows[b][j] @ rows[b][j]))
    cache, _ = fill_pools(st, [r[:, None] for r in rows], [r[:, None, :1] for r in rows], page, n_pages, dtype)
    gate = dev(rng.standard_normal((T, H + 9)) * 2, dtype)[:, 9:]
    out = torch.full((T, H * rank), float("nan"), dtype=dtype, device="cuda")
    want = np.zeros((T, H, rank))
    qd = dev(qa.reshape(T, -1))
    qr = host(dev(qa, BF16)) if ops.latent_attention_queries_dtype(st, dtype, dk, rank) == BF16 else host(dev(qa))
    ops.launches_by_kernel.clear()
    ops.attention_latent(qd, cache, out, st, 0, H, rank, page, scale, None, window, gate=gate)
    for t in range(T):
        b, pos = st.host_seq[t], st.host_pos[t]
        lo = max(0, pos - window + 1) if window else 0
        for h in range(H):
            want[t, h] = P.softmax(rows[b][lo:pos + 1] @ qr[t, h] * scale) @ rows[b][lo:pos + 1, :rank]
    want *= P.sigmoid(host(gate))[:, :, None]
    np.testing.assert_allclose(host(out).reshape(T, H, rank), want, rtol=0, atol=3e-5 if dtype == torch.float32 else 0.04)
    if dtype == BF16 and ops.latent_attention_takes_mma(dtype, dk, rank):
        assert ops.launches_by_kernel.get("attention_latent.decode.mma" + (".cluster" if window == 0 or window >= 256 else ""))


@pytest.mark.parametrize("H,G,d,dv", [(2, 1, 64, 128), (1, 1, 40, 56)])
def test_a_single_token_far_into_a_long_context(H, G, d, dv):
    """More pieces than a cluster holds: they are merged by a second kernel."""
    from rust_llm_inference_server_b200 import ops
    rng = np.random.default_rng(d)
    page, ctx = 64, [20000, 300]
    st = hand_step(ctx, [1, 1], page, 330, rng)
    keys, vals = [rng.standard_normal((c, G, 2 * d)) for c in ctx], [rng.standard_normal((c, G, dv)) for c in ctx]
    q = rng.standard_normal((2, H, 2, d))
    for h in range(H):                                      # a key in the first piece and one in the middle
        for m, j in ((0, 3), (1, 11111)):
            k = keys[0][j, h // (H // G), m * d:(m + 1) * d]
            q[0, h, m] = k * (11.0 / 0.1 / float(k @ k))
    q = dev(q.reshape(2, -1), BF16)
    kr, vr = [host(dev(k, BF16)) for k in keys], [host(dev(v, BF16)) for v in vals]
    kc, vc = (torch.full((330, G, page, w), 50.0, dtype=BF16, device="cuda") for w in (2 * d, dv))
    for b, (k, v) in enumerate(zip(kr, vr)):
        for p in range(0, ctx[b], page):
            for pool, x in ((kc, k), (vc, v)):
                part = dev(x[p:p + page], BF16).transpose(0, 1)
                pool[int(st.host_tables[b, p // page]), :, :part.shape[1]] = part
    out = torch.full((2, H * dv), float("nan"), dtype=BF16, device="cuda")
    ops.launches_by_kernel.clear()
    ops.attention_difference(q, kc, vc, out, None, st, 0, H, G, d, dv, page, 0.1, 50.0, 0.5, 0.7, 1e-5)
    want = plain_difference_rows(host(q).reshape(2, H, 2, d), [k.reshape(-1, G, 2, d) for k in kr], vr, 0.1, 50.0, 0, 0.5, 0.3, 1e-5,
                                 np.full((2, H), 60.0), st, H, G)
    np.testing.assert_allclose(host(out).reshape(2, H, dv), want, rtol=0, atol=0.05)
    assert ops.launches_by_kernel == {"attention_difference.decode.mma.split": 1}


@pytest.mark.parametrize("T,H,N,K", [(1, 3, 40, 16), (8, 6, 64, 32), (16, 16, 512, 128), (9, 2, 24, 512), (5, 16, 128, 512), (3, 1, 10, 264),
                                     (16, 5, 72, 200)])
def test_small_product_a_head(T, H, N, K):
    from rust_llm_inference_server_b200 import ops
    rng = np.random.default_rng(N + K)
    wide = dev(rng.standard_normal((T, H * (K + 8) + 16)), BF16)
    a = wide[:, 8:8 + H * (K + 8)].unflatten(1, (H, K + 8))[:, :, :K]                # slices of wider rows
    w = dev(rng.standard_normal((H, N, K)) / np.sqrt(K), BF16)
    out = torch.full((T, H, N + 3), 7.0, dtype=BF16, device="cuda")
    ops.launches_by_kernel.clear()
    ops.per_head_linear(a, w, out[:, :, :N])
    assert ops.launches_by_kernel == {"per_head_small": 1}
    np.testing.assert_allclose(host(out[:, :, :N]), np.einsum("thk,hnk->thn", host(a), host(w)), rtol=1e-2, atol=0.02)
    assert float((out[:, :, N:].float() - 7.0).abs().max()) == 0.0


@pytest.mark.parametrize("T,H,d,rank,rot", [(1, 3, 16, 64, 16), (8, 16, 128, 512, 64), (16, 6, 32, 128, 32), (5, 2, 8, 64, 0)])
def test_latent_rows_and_folded_queries_in_one_launch(T, H, d, rank, rot):
    """Against the operations one by one: the same rows in the cache and nothing beside them, the same queries."""
    from rust_llm_inference_server_b200 import ops
    rng = np.random.default_rng(T + d)
    page = 16
    ctx = [int(c) for c in rng.integers(1, 60, size=T)]
    st = hand_step(ctx, [1] * T, page, 4 * T + 2, rng)
    n_q = H * (d + rot)
    proj = dev(rng.standard_normal((T, n_q + rank + rot + 8)), BF16)
    q, z = proj[:, :n_q], proj[:, n_q:n_q + rank + rot]
    fold, w = dev(rng.standard_normal((H, rank, d)) / np.sqrt(d), BF16), dev(1 + 0.2 * rng.standard_normal(rank))
    freq = dev(100.0 ** (-2.0 * np.arange(rot // 2) / max(rot, 1)))
    caches = [torch.full((4 * T + 2, 1, page, rank + rot), 7.0, dtype=BF16, device="cuda") for _ in range(2)]
    qas = [torch.empty((T, H * (rank + rot)), dtype=BF16, device="cuda") for _ in range(2)]
    assert ops.latent_step_takes(q, BF16, fold, H, d, rot)
    ops.latent_step(q, z, fold, w, 1e-5, freq, rot, 1.0, st.positions, st.slots[0], caches[0], qas[0], H, d, rank, page)
    ops.latent_kv_store(z, w, 1e-5, freq, rot, 1.0, st.positions, st.slots[0], caches[1], rank, page)
    torch.bmm(q.unflatten(1, (H, d + rot))[:, :, :d].transpose(0, 1), fold.transpose(1, 2), out=qas[1].view(T, H, -1)[:, :, :rank].transpose(0, 1))
    if rot:
        ops.latent_q_rope(q, qas[1], freq, rot, 1.0, st.positions, H, d, rot, rank)
    assert torch.equal(caches[0], caches[1])
    np.testing.assert_allclose(host(qas[0]), host(qas[1]), rtol=1e-2, atol=0.02)
    before = caches[0].clone()
    ops.latent_step(q, z, fold, w, 1e-5, freq, rot, 1.0, st.positions, None, caches[0], qas[0], H, d, rank, page)
    assert torch.equal(caches[0], before)


# ---- whole models ------------------------------------------------------------------------------

ALONE = {
    "attention_only": U.model(61, 48, 1e-5, [U.attention(4, 2, 16, 8, 0.5, 8.0, 0.3, (8, 100.0))]),
    "latent_only": U.model(61, 48, 1e-5, [U.latent(3, 8, 8, 12, 16, 0.4, 11, 200.0)]),
    "attention_with_unit": U.model(61, 48, 1e-5, [U.attention(2, 2, 24, 24, 0.3, 20.0, 0.7, (24, 1000.0), 40)]),
    "latent_with_unit": U.model(61, 48, 1e-5, [U.latent(2, 16, 4, 8, 24, 0.4, 30, 200.0, 56)]),
    "looped": U.model(61, 48, 1e-5, [U.attention(2, 1, 8, 8, 0.6, 9.0, 0.2, (4, 50.0), 24)], (0, 1, 3)),
    "loop_at_the_end": U.model(61, 48, 1e-5, [U.latent(2, 8, 8, 8, 16, 0.5, 5, 90.0), U.latent(2, 8, 8, 8, 16, 0.5, 5, 90.0, 32)], (1, 2, 2)),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", sorted(ALONE))
def test_each_kind_of_layer_alone(model_root, which, dtype):
    d = U.make_dir(model_root, which, ALONE[which], 11)
    reqs = requests_for(ALONE[which], [1, 2, 37, 90])
    ref = plain_logits(d, reqs, dtype)
    for fam, steps in (("whole", R.whole_trace(reqs)), ("decode", R.decode_trace(reqs, tail=20)),
                       ("chunks", R.chunk_trace(reqs, seed=2))):
        s = session(d, dtype, R.live_token_peak(steps), 8)
        ok, what = ref.holds(R.collect(s.step, steps))
        assert ok, f"{which} {dtype} {fam}: {what}"


@pytest.mark.parametrize("which", ["A", "D", "E"])
def test_the_stream_after_every_run_of_a_layer(model_root, which):
    from rust_llm_inference_server_b200.parts.block import ParallelBlock
    d = U.make_dir(model_root, which)
    cfg, w = U.read_config(d), U.plain_weights(d)
    toks = requests_for(cfg, [45], seed=4)["r0"]
    want = P.forward(cfg, w, toks)[1]
    s = session(d, "float32", 64, 16)
    seen = []
    for blk in set(s.model.blocks):
        assert isinstance(blk, ParallelBlock)

        def tapped(*a, _inner=blk.forward, **k):
            resid, pending = _inner(*a, **k)
            seen.append(host(resid) + sum(host(p) for p in (pending if isinstance(pending, tuple) else (pending,))))
            return resid, pending
        blk.forward = tapped
    s.step({"step": 0, "entries": [{"id": "x", "tokens": toks, "want": [len(toks) - 1]}], "end": ["x"]})
    assert len(seen) == len(U.runs(cfg))
    for i, (got, ref) in enumerate(zip(seen, want)):
        np.testing.assert_allclose(got, ref, rtol=0, atol=2e-4 * max(1.0, np.abs(ref).max() / 10), err_msg=f"after run {i}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which,page,lens", [("A", 16, [1, 50, 97, 200, 64, 17, 2]), ("A", 8, [130, 33, 2, 71, 40]),
                                             ("B", 16, [3, 150, 40, 2, 129, 1]), ("C", 16, [1, 70, 333, 2, 129, 64, 65]),
                                             ("C", 64, [200, 65, 2, 30]), ("D", 16, [90, 1, 33, 150, 2]), ("D", 32, [260, 31, 5, 90]),
                                             ("E", 16, [420, 3, 200, 77]), ("F", 16, [300, 5, 131, 64])])
def test_all_ways_of_cutting_give_the_plain_logits(model_root, which, page, lens, dtype):
    from rust_llm_inference_server_b200 import ops
    ops.launches_by_kernel.clear()
    d = U.make_dir(model_root, which)
    reqs = requests_for(U.CONFIGS[which], lens, seed=page)
    ref = plain_logits(d, reqs, dtype)
    families = {
        "whole": (R.whole_trace(reqs), 4),
        "decode": (R.decode_trace(reqs, tail=40), 4),
        "chunks": (R.chunk_trace(reqs, seed=3), 4),
        "mixed": (R.mixed_trace(reqs, seed=4), 4),
        "mixed2": (R.mixed_trace(dict(reversed(list(reqs.items()))), seed=5, max_live=2), 2),
    }
    results = {}
    for fam, (steps, live) in families.items():
        s = session(d, dtype, R.live_token_peak(steps, max(64, page)), page, max_live=live)
        for pool in s.storage.pools:                         # whatever a page held before must not matter
            for t in (pool if isinstance(pool, tuple) else (pool,)):
                t.fill_(30.0)
        results[fam] = R.collect(s.step, steps)
        assert s.cache.check_invariants() == ""
        for g in range(len(s.storage.groups)):
            assert s.cache.num_free_pages(g) == s.cache.group(g).num_pages, fam
        ok, what = ref.holds(results[fam])
        assert ok, f"{which} {dtype} {fam} vs plain: {what}"
    for fam in ("decode", "chunks", "mixed", "mixed2"):
        ok, what = ref.holds(results[fam], results["whole"], between=True)
        assert ok, f"{which} {dtype}: {fam} differs from whole by {what}"
    launched = ops.launches_by_kernel
    needed = {"layer_norm", "layer_norm.rows", "qk_norm_store.rot", "latent_kv_store"}
    if dtype == "float32":
        needed |= {"attention_difference", "attention_latent"}
    elif U.CONFIGS[which]["width"] % 8 == 0:
        needed |= {"stream_gemm.scaled.centred.mixed", "stream_gemm.sink.centred.two", "embedding.sink"}
        if U.CONFIGS[which].get("loop"):
            needed |= {"stream_gemm.sink.centred"}
        if which != "F":
            needed |= {"attention_difference.decode.mma.cluster" if max(lens) > 190 else "attention_difference.decode.mma",
                       "attention_difference.prefill.tcgen05"}
        if which in ("C", "E"):
            needed |= {"attention_latent.decode.mma", "attention_latent.prefill.mma", "gemm_tcgen05.glu4", "latent_step", "per_head_small"}
    assert needed <= set(launched), f"never launched {sorted(needed - set(launched))}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which,n,tail", [("A", 230, 215), ("C", 260, 240)])
def test_long_decoding_while_the_windows_pass_over_decoded_tokens(model_root, which, n, tail, dtype):
    d = U.make_dir(model_root, which)
    reqs = requests_for(U.CONFIGS[which], [n], seed=9)
    ref = plain_logits(d, reqs, dtype)
    steps = R.decode_trace(reqs, tail=tail)             # a page border every 8 tokens; steps replayed from a CUDA graph
    s = session(d, dtype, R.live_token_peak(steps), 8)
    ok, what = ref.holds(R.collect(s.step, steps))
    assert ok, what
    assert s.runner._graph_launches > 0


def test_pages_behind_a_window_are_given_back(model_root):
    d = U.make_dir(model_root, "A")
    s = session(d, "bfloat16", 256, 8, max_live=1)
    toks = requests_for(U.CONFIGS["A"], [180], seed=2)["r0"]
    s.step({"step": 0, "entries": [{"id": "x", "tokens": toks[:100], "want": []}], "end": []})
    for i in range(100, 180):
        s.step({"step": i, "entries": [{"id": "x", "tokens": toks[i:i + 1], "want": []}], "end": []})
    held = {(g.spec.window if hasattr(g, "spec") else None): s.cache.group(i).num_pages - s.cache.num_free_pages(i)
            for i, g in enumerate(s.storage.groups)}
    assert min(held.values()) <= 3 and max(held.values()) >= 180 // 8      # a window of 7 holds two or three pages of 8


def plain_greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(np.argmax(P.forward(cfg, w, toks)[0][-1])))
    return toks[len(prompt):]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_entry_point(model_root, dtype):
    """Prompts of unequal length batched by the scheduler, portions of 16 tokens, decode steps from CUDA graphs and
    launched ahead; two seats, so the later prompts take over pages."""
    from rust_llm_inference_server_b200 import LLM, SamplingParams
    d = U.make_dir(model_root, "A")
    cfg, w = U.read_config(d), U.plain_weights(d)
    prompts = list(requests_for(cfg, [1, 9, 40, 23, 3], seed=12).values())
    llm = LLM(d, dtype=dtype, max_seq_len=128, num_blocks=60, block_size=8, max_num_seqs=2, max_batched_tokens=16)
    outs = llm.generate(prompts, SamplingParams(max_tokens=12))
    for p, o in zip(prompts, outs):
        want = plain_greedy(cfg, w, p, 12)
        assert o.finish_reason == "length" and len(o.token_ids) == 12
        if o.token_ids != want:
            i = next(k for k, (a, b) in enumerate(zip(o.token_ids, want)) if a != b)
            lg = P.forward(cfg, w, p + want[:i])[0][-1]
            gap = (lg[want[i]] - lg[o.token_ids[i]]) / lg.std()
            assert dtype == "bfloat16" and gap < 0.15, f"parted at token {i} with a gap of {gap}"
    assert llm.engine.cache.check_invariants() == ""
    assert llm.engine.runner._graph_launches > 0


def test_command_line_serves_the_design(tmp_path):
    """random-weights and generate of the command line with a Dotivik folder."""
    import json
    import os
    import subprocess
    import sys
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))

    def rlis(*args):
        return subprocess.run([sys.executable, os.path.join(root, "bin", "rlis"), *args], capture_output=True,
                              text=True, timeout=600)

    cfg_file = tmp_path / "c.json"
    cfg_file.write_text(json.dumps(U.CONFIGS["A"]))
    d = str(tmp_path / "m")
    r = rlis("random-weights", "--config", str(cfg_file), "--seed", "21", "--out", d)
    assert r.returncode == 0, r.stderr[-2000:]
    cfg, w = U.read_config(d), U.plain_weights(d)
    assert cfg["architecture"] == "Dotivik" and set(w) == set(U.tensor_shapes(cfg))
    prompt = [5, 9, 200, 31, 7]
    r = rlis("generate", "--model", d, "--dtype", "f32", "--prompt-ids", ",".join(map(str, prompt)),
             "--max-tokens", "8", "--max-seq-len", "64", "--kv-cache-gb", "0.001", "--block-size", "8",
             "--max-num-seqs", "2")
    assert r.returncode == 0, r.stderr[-2000:]
    assert [int(t) for t in r.stdout.split()] == plain_greedy(cfg, w, prompt, 8)
