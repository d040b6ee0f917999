"""Papulix on the GPU against the plain restatement: every kernel alone (the streams' update and norm, also inside the
streaming product; the delta rule with a decay a channel and the state-space recurrence cut into portions over slots that
held something else; norms over whole projections and the paged write; attention with one added to the softmax's
denominator under a gate a channel, with a key far back and at page borders made to carry a head's weight; the gate before
a norm in parts; gated units with biases through each of their products), every kind of layer alone in a small model, the
streams' sum after every run of a layer, whole prompts against portions, single tokens and mixed batches in pools so small
that pages and slots are used again, long decoding, and greedy generation through the entry point and the command line."""

from types import SimpleNamespace

import numpy as np
import pytest
import torch

from tests import papulix_util as U
from tests import replay_util as R
from tests.plain import papulix_plain as P
from tests.test_gavodra_gpu import dev, fill_pools, hand_step, host, position_error, requests_for
from tests.test_lanirax_gpu import RECURRENCE_SCHEDULES
from tests.test_rumedra_gpu import Limits, jittered_bfloat16, to_bfloat16

pytestmark = pytest.mark.gpu

# A position's error and its limits are those of the Rumedra tests: float32 a fixed part of the logits' spread, bfloat16
# three times what rounding the products' inputs does at that position in the plain restatement, and no less than FLOOR.
FLOOR = 0.03
BF16 = torch.bfloat16


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


def stream_case(rng, S, T, W, dtype):
    return SimpleNamespace(x=rng.standard_normal((T, S, W)) * 2, y=host(dev(rng.standard_normal((T, W)) * 2, dtype)),
                           bias=rng.standard_normal(W), mix=np.eye(S) * 0.7 + 0.4 * rng.standard_normal((S, S)),
                           write=1 + 0.5 * rng.standard_normal(S), read=rng.standard_normal(S),
                           w=1 + 0.3 * rng.standard_normal(W), b=0.5 * rng.standard_normal(W), alpha=0.8)


def plain_streams(c, x=None):
    """(new streams [T, S, W], h of the streams read by c.read under the dynamic tanh)."""
    x = c.x if x is None else x
    new = P.stream_update(x.transpose(1, 0, 2), c.mix, c.write, c.y + c.bias)
    h = P.dynamic_tanh(P.stream_input(new, c.read), {"n": c.w, "n.b": c.b, "n.alpha": c.alpha}, "n")
    return new.transpose(1, 0, 2), h


@pytest.mark.parametrize("dtype", [torch.float32, BF16])
@pytest.mark.parametrize("S,T,W", [(1, 3, 40), (2, 7, 96), (3, 5, 1030), (4, 2, 2048), (5, 600, 36), (8, 1, 77)])
def test_streams_are_updated_at_once_and_normed(dtype, S, T, W):
    from rust_llm_inference_server_b200 import ops
    rng = np.random.default_rng(S * W)
    c = stream_case(rng, S, T, W, dtype)
    f = lambda a: dev(a)
    tol = 2e-5 if dtype == torch.float32 else 0.02
    norm = ops.StreamNorm("dynamic_tanh", f(c.w), f(c.b), c.alpha)
    update = dict(y=dev(c.y, dtype), y_bias=f(c.bias), mix=f(c.mix), out_coef=f(c.write))
    x, h = f(c.x), torch.empty((T, W), dtype=dtype, device="cuda")
    new, want = plain_streams(c)
    ops.stream_mix(x, S, x_out=x, in_coef=f(c.read), norm=norm, h=h, **update)                 # in place
    np.testing.assert_allclose(host(x), new, rtol=0, atol=2e-5)
    np.testing.assert_allclose(host(h), want, rtol=0, atol=tol)
    # rows only: the streams stay as they are
    rows = rng.integers(0, T, size=4)
    x, h4 = f(c.x), torch.empty((4, W), dtype=dtype, device="cuda")
    ops.stream_mix(x, S, in_coef=f(c.read), norm=norm, h=h4, rows=dev(rows, torch.int32), **update)
    assert torch.equal(x, f(c.x))
    np.testing.assert_allclose(host(h4), want[rows], rtol=0, atol=tol)
    # one row that is every stream, into streams of its own; the plain sum in float32
    base = c.x[:, 0]
    home, u = torch.full((T, S, W), float("nan"), device="cuda"), torch.empty((T, W), device="cuda")
    ops.stream_mix(f(base), S, x_out=home, u_out=u, **update)
    new1, _ = plain_streams(c, np.repeat(base[:, None], S, axis=1))
    np.testing.assert_allclose(host(home), new1, rtol=0, atol=2e-5)
    np.testing.assert_allclose(host(u), new1.sum(axis=1), rtol=0, atol=5e-5)
    # nothing to join, no norm; and a norm with a mean square
    ops.stream_mix(f(c.x), S, in_coef=f(c.read), h=h)
    np.testing.assert_allclose(host(h), np.einsum("s,tsw->tw", c.read, c.x), rtol=1e-2 if dtype == BF16 else 0, atol=max(tol, 2e-5))
    ops.stream_mix(x, S, x_out=x, in_coef=f(c.read), norm=ops.StreamNorm("rmsnorm", f(c.w), eps=1e-3), h=h, **update)
    np.testing.assert_allclose(host(x), new, rtol=0, atol=2e-5)
    want = P.rms_norm(np.einsum("s,tsw->tw", c.read, new), c.w, 1e-3)
    np.testing.assert_allclose(host(h), want, rtol=1e-2 if dtype == BF16 else 0, atol=tol)
    # the ordinary residual addition and its norm: one stream, no coefficients
    r, d = f(base), dev(c.y, dtype)
    ops.stream_mix(r, 1, y=d, x_out=r.unsqueeze(1), norm=norm, h=h)
    np.testing.assert_allclose(host(r), base + c.y, rtol=0, atol=1e-5)
    np.testing.assert_allclose(host(h), np.tanh(c.alpha * (base + c.y)) * c.w + c.b, rtol=0, atol=tol)


@pytest.mark.parametrize("S,M,N,K", [(1, 1, 96, 40), (2, 8, 320, 512), (3, 16, 200, 64), (4, 5, 2048, 2048), (8, 3, 1000, 776)])
def test_streaming_product_into_the_streams(S, M, N, K):
    """The product's epilogue against the kernel of its own: the same streams and the same rows."""
    from rust_llm_inference_server_b200 import ops
    rng = np.random.default_rng(N + K)
    c = stream_case(rng, S, M, N, BF16)
    wide = dev(rng.standard_normal((M, K + 24)), BF16)
    w = dev(rng.standard_normal((N, K)) / np.sqrt(K), BF16)
    norm = ops.StreamNorm("dynamic_tanh", dev(c.w), dev(c.b), c.alpha)
    for x in (wide[:, :K].contiguous(), wide[:, 8:8 + K]):                       # whole rows and a column slice
        y = ops.stream_gemm(x, w)
        for bias in (dev(c.bias), None):
            for old in (dev(c.x), dev(c.x[:, 0])):
                for read in (dev(c.read), None):
                    want_x, want_h = torch.empty((M, S, N), device="cuda"), torch.empty((M, N), dtype=BF16, device="cuda")
                    ops.stream_mix(old, S, y=y, y_bias=bias, mix=dev(c.mix), out_coef=dev(c.write), x_out=want_x, in_coef=read,
                                   norm=norm, h=want_h)
                    got_x = torch.full((M, S, N), float("nan"), device="cuda") if old.dim() == 2 else old
                    sink = ops.StreamsSink(old, got_x, S, dev(c.mix), dev(c.write), read, norm)
                    h = ops.linear(x, w, sink=sink, bias=bias)
                    np.testing.assert_allclose(host(got_x), host(want_x), rtol=0, atol=2e-5)
                    np.testing.assert_allclose(host(h), host(want_h), rtol=0, atol=0.02)
    assert ops.launches_by_kernel.get("stream_gemm.streams")
    ops.check_device_errors()


@pytest.mark.parametrize("M", [1, 9, 16, 30, 50, 100])
def test_streaming_product_with_a_bias(M):
    from rust_llm_inference_server_b200 import ops
    rng = np.random.default_rng(M)
    N, K = 264, 328
    x, w, b = dev(rng.standard_normal((M, K)), BF16), dev(rng.standard_normal((N, K)) / np.sqrt(K), BF16), dev(rng.standard_normal(N))
    want = host(x) @ host(w).T + host(b)
    np.testing.assert_allclose(host(ops.stream_gemm(x, w, torch.float32, bias=b)), want, rtol=0, atol=1e-4)
    np.testing.assert_allclose(host(ops.stream_gemm(x, w, bias=b)), want, rtol=1e-2, atol=1e-2)
    g, u = want.reshape(M, -1, 2, 4)[:, :, 0].reshape(M, -1), want.reshape(M, -1, 2, 4)[:, :, 1].reshape(M, -1)
    np.testing.assert_allclose(host(ops.stream_gemm(x, w, swiglu4=True, bias=b)), P.silu(g) * u, rtol=1e-2, atol=1e-2)
    if M <= 16:
        nw, r = dev(rng.standard_normal(N)), dev(rng.standard_normal((M, N)))
        before = host(r)
        rows = ops.stream_gemm(x, w, sink=ops.ResidualSink(r, nw, 1e-5), bias=b)
        np.testing.assert_allclose(host(r), before + want, rtol=0, atol=0.02)
        np.testing.assert_allclose(host(rows.x), host(r) * host(nw), rtol=1e-2, atol=1e-2)


@pytest.mark.parametrize("dtype", [torch.float32, BF16])
@pytest.mark.parametrize("M,K,off", [(3, 24, 8), (40, 16, 0), (200, 48, 24), (5, 20, 3)])
def test_products_over_a_column_slice(dtype, M, K, off):
    from rust_llm_inference_server_b200 import ops
    rng = np.random.default_rng(M)
    wide, w = dev(rng.standard_normal((M, 88)), dtype), dev(rng.standard_normal((96, K)), dtype)
    got = ops.linear(wide[:, off:off + K], w)
    np.testing.assert_allclose(host(got), host(wide)[:, off:off + K] @ host(w).T, rtol=1e-2 if dtype == BF16 else 0,
                               atol=0.05 if dtype == BF16 else 1e-4)


def run_schedule(portions, lens_rows, state_floats, launch, nh, dv, dtype):
    """Feeds the schedule's portions of every request's rows through `launch(step, [row arrays of the step], out)`; yields
    (request, first row, rows of the result)."""
    lens, schedule = RECURRENCE_SCHEDULES[portions]
    rng = np.random.default_rng(5)
    state = torch.full((3, state_floats), 30.0, dtype=torch.float32, device="cuda")
    free, slot_of, done = [2, 0, 1], {}, {r: 0 for r in range(len(lens))}
    for entries in schedule:
        for r, _ in entries:
            if r not in slot_of:
                slot_of[r] = free.pop()
        ctx = [done[r] + n for r, n in entries]
        st = hand_step(ctx, [n for _, n in entries], 16, sum(-(-c // 16) for c in ctx) + 1, rng)
        st.state_slots = dev([slot_of[r] for r, _ in entries], torch.int32)
        rows = [dev(np.concatenate([rows[r][done[r]:done[r] + n] for r, n in entries]), dtype) for rows in lens_rows]
        out = torch.full((st.n_tokens, nh * dv), float("nan"), dtype=torch.float32, device="cuda")
        launch(st, rows, state, out, st.n_tokens > 4 * st.n_seqs)
        got, at = host(out).reshape(-1, nh, dv), 0
        for r, n in entries:
            yield r, done[r], got[at:at + n]
            at += n
            done[r] += n
            if done[r] == lens[r]:
                free.append(slot_of[r])
    assert done == dict(enumerate(lens))


def plain_channel_delta_rows(x, b, a, taps, a_log, dt_bias, nh, nqk, d, dv):
    T = x.shape[0]
    y = P.short_conv(x, taps)
    q, k, v = y[:, :nqk * d].reshape(T, nqk, d), y[:, nqk * d:2 * nqk * d].reshape(T, nqk, d), y[:, 2 * nqk * d:].reshape(T, nh, dv)
    q = q / np.sqrt((q * q).sum(-1, keepdims=True) + 1e-6) * d ** -0.5
    k = k / np.sqrt((k * k).sum(-1, keepdims=True) + 1e-6)
    g = np.exp(-np.exp(a_log)[None, :, None] * P.softplus(a + dt_bias).reshape(T, nh, d))
    beta = P.sigmoid(b)
    return np.stack([P.channel_decay_delta(q[:, h // (nh // nqk)], k[:, h // (nh // nqk)], v[:, h], beta[:, h], g[:, h])
                     for h in range(nh)], axis=1)


@pytest.mark.parametrize("dtype", [torch.float32, BF16])
@pytest.mark.parametrize("portions", ["long", "short"])
@pytest.mark.parametrize("nh,nqk,d,dv,taps,harsh", [(4, 2, 16, 24, 3, 0), (1, 1, 8, 16, 1, 0), (3, 1, 24, 16, 5, 1),
                                                    (2, 1, 64, 32, 4, 0), (4, 4, 32, 64, 4, 1), (6, 3, 12, 20, 4, 0),
                                                    (2, 2, 128, 128, 2, 0), (2, 1, 200, 40, 8, 0), (2, 1, 300, 16, 2, 0),
                                                    (1, 1, 30, 7, 4, 0)])
def test_channel_decay_cut_into_portions_over_slots_that_held_something_else(dtype, portions, nh, nqk, d, dv, taps, harsh):
    """Six requests over three state slots that start full of junk: portions of one and two tokens beside long ones,
    requests that sit out a step, a slot taken over by a new request in the step after its owner ended.  Every output row
    against the plain recurrence over the whole request.  `harsh`: some channels forget everything at every token (a decay
    that is zero in float32) beside channels that forget nothing."""
    from rust_llm_inference_server_b200 import ops
    rng = np.random.default_rng(d * 7 + taps)
    lens, _ = RECURRENCE_SCHEDULES[portions]
    ops.launches_by_kernel.clear()
    C, lead, gap = 2 * nqk * d + nh * dv, 8, 5
    b_off = lead + C + gap
    N = -(-(b_off + nh) // 8) * 8
    rows = [host(dev(rng.standard_normal((n, N)) * 1.5, dtype)) for n in lens]      # what the kernel reads, exactly
    dec = [host(dev(rng.standard_normal((n, nh * d + 3)) * 2.0, dtype)) for n in lens]
    taps_w = dev(rng.standard_normal((C, taps)) * 0.6 + 0.3)
    a_log, dt_bias = dev(rng.uniform(-2.5, 0.5, nh)), rng.uniform(-1.0, 1.0, nh * d)
    if harsh:
        dt_bias[::3], dt_bias[1::3] = 300.0, -200.0
    dt_bias = dev(dt_bias)
    want = [plain_channel_delta_rows(r[:, lead:lead + C], r[:, b_off:b_off + nh], a[:, 2:2 + nh * d], host(taps_w), host(a_log),
                                     host(dt_bias), nh, nqk, d, dv) for r, a in zip(rows, dec)]

    def launch(st, arrays, state, out, chunks):
        ops.channel_delta(arrays[0], lead, b_off, arrays[1][:, 2:2 + nh * d], taps_w, a_log, dt_bias, state, out, st, nh, nqk, d,
                          dv, taps, 1e-6, d ** -0.5, chunks=chunks)
    worst = max(float(np.abs(got - want[r][at:at + len(got)]).max()) for r, at, got in run_schedule(
        portions, [rows, dec], ops.conv_recurrence_state_floats(nh, nqk, d, dv, taps), launch, nh, dv, dtype))
    assert worst <= 5e-5, worst
    assert ops.launches_by_kernel.get("channel_delta.scan")
    assert bool(ops.launches_by_kernel.get("channel_delta.chunks")) == (portions == "long")
    # the test bites: without the state, or with one decay for all channels of a head, the later rows differ
    if portions == "long" and not harsh and d <= 200:
        cut = plain_channel_delta_rows(rows[3][10:, lead:lead + C], rows[3][10:, b_off:b_off + nh], dec[3][10:, 2:2 + nh * d],
                                       host(taps_w), host(a_log), host(dt_bias), nh, nqk, d, dv)
        assert np.abs(want[3][10:] - cut).max() > 0.02
        flat = dec[3][:, 2:2 + nh * d].reshape(-1, nh, d).mean(-1, keepdims=True).repeat(d, -1).reshape(-1, nh * d)
        one = plain_channel_delta_rows(rows[3][:, lead:lead + C], rows[3][:, b_off:b_off + nh], flat, host(taps_w), host(a_log),
                                       host(dt_bias), nh, nqk, d, dv)
        assert np.abs(want[3] - one).max() > 0.02
    ops.check_device_errors()


def plain_state_space_rows(x, b, taps, conv_b, a_log, dt_bias, skip, nh, groups, n, dv):
    T, inner = x.shape[0], nh * dv
    y = P.short_conv(x, taps, conv_b)
    v, B, C = y[:, :inner].reshape(T, nh, dv), y[:, inner:inner + groups * n].reshape(T, groups, n), y[:, inner + groups * n:].reshape(T, groups, n)
    dt = P.softplus(b + dt_bias)
    return np.stack([P.state_space(v[:, h], B[:, h // (nh // groups)], C[:, h // (nh // groups)], dt[:, h], -np.exp(a_log[h]), skip[h])
                     for h in range(nh)], axis=1)


@pytest.mark.parametrize("dtype", [torch.float32, BF16])
@pytest.mark.parametrize("portions", ["long", "short"])
@pytest.mark.parametrize("nh,groups,n,dv,taps,bias", [(4, 2, 16, 24, 3, True), (1, 1, 8, 16, 1, True), (3, 1, 24, 16, 5, False),
                                                      (8, 2, 64, 32, 4, True), (6, 3, 20, 10, 4, True), (2, 1, 128, 64, 2, True),
                                                      (2, 2, 200, 40, 8, True), (1, 1, 300, 16, 2, True), (5, 5, 30, 7, 4, True)])
def test_state_space_cut_into_portions_over_slots_that_held_something_else(dtype, portions, nh, groups, n, dv, taps, bias):
    from rust_llm_inference_server_b200 import ops
    rng = np.random.default_rng(n * 7 + taps)
    lens, _ = RECURRENCE_SCHEDULES[portions]
    ops.launches_by_kernel.clear()
    C, lead, gap = nh * dv + 2 * groups * n, 8, 3
    b_off = lead + C + gap
    N = -(-(b_off + nh) // 8) * 8
    rows = [host(dev(rng.standard_normal((k, N)) * 1.2, dtype)) for k in lens]
    taps_w = dev((rng.standard_normal((C, taps)) * 0.6 + 0.3) / np.sqrt(np.sqrt(n)))
    conv_b = dev(0.5 * rng.standard_normal(C)) if bias else None
    a_log, dt_bias, skip = dev(rng.uniform(-3.5, 0.5, nh)), dev(rng.uniform(-2.0, 0.5, nh)), dev(rng.standard_normal(nh))
    args = (host(taps_w), host(conv_b) if bias else None, host(a_log), host(dt_bias), host(skip), nh, groups, n, dv)
    want = [plain_state_space_rows(r[:, lead:lead + C], r[:, b_off:b_off + nh], *args) for r in rows]

    def launch(st, arrays, state, out, chunks):
        ops.state_space(arrays[0], lead, b_off, taps_w, conv_b, a_log, dt_bias, skip, state, out, st, nh, groups, n, dv, taps,
                        chunks=chunks)
    worst = max(float((np.abs(got - want[r][at:at + len(got)]).max() / max(1.0, np.abs(want[r]).max())))
                for r, at, got in run_schedule(portions, [rows], ops.conv_recurrence_state_floats(nh, groups, n, dv, taps), launch,
                                               nh, dv, dtype))
    assert worst <= 2e-5, worst
    assert ops.launches_by_kernel.get("state_space.scan")
    assert bool(ops.launches_by_kernel.get("state_space.chunks")) == (portions == "long")
    if portions == "long":                               # the test bites: without the state the later rows differ
        cut = plain_state_space_rows(rows[3][10:, lead:lead + C], rows[3][10:, b_off:b_off + nh], *args)
        assert np.abs(want[3][10:] - cut).max() > 0.05
    ops.check_device_errors()


@pytest.mark.parametrize("dtype", [torch.float32, BF16])
@pytest.mark.parametrize("T,W,groups", [(3, 96, 2), (5, 60, 3), (2, 4096, 1), (9, 24, 24), (4, 70, 5), (2, 9216, 1), (3, 512, 4)])
def test_gate_before_a_norm_in_parts(dtype, T, W, groups):
    from rust_llm_inference_server_b200 import ops
    rng = np.random.default_rng(W)
    x, w = dev(rng.standard_normal((T, W)) * 3), dev(1 + 0.3 * rng.standard_normal(W))
    z = dev(rng.standard_normal((T, W + 12)) * 2, dtype)[:, 4:4 + W]
    out = torch.empty((T, W), dtype=dtype, device="cuda")
    ops.gate_group_norm(x, z, w, 1e-3, out, groups)
    want = P.gated_group_norm(host(x), host(z), host(w), groups, 1e-3)
    np.testing.assert_allclose(host(out), want, rtol=1e-2 if dtype == BF16 else 0, atol=2e-5 if dtype == torch.float32 else 0.02)


@pytest.mark.parametrize("dtype", [torch.float32, BF16])
@pytest.mark.parametrize("H,G,d,dv", [(4, 2, 16, 24), (1, 1, 8, 8), (5, 5, 20, 12), (8, 1, 128, 96), (6, 3, 64, 32), (32, 8, 64, 64)])
def test_norm_over_whole_projections_and_the_paged_write(dtype, H, G, d, dv):
    """Queries and keys normed over all their heads together; portions that start in the middle of a page; nothing else of
    the pools is written."""
    from rust_llm_inference_server_b200 import ops
    rng = np.random.default_rng(d + H)
    page, n_pages = 8, 40
    st = hand_step([119, 5, 30], [7, 1, 30], page, n_pages, rng)
    T, lead = st.n_tokens, 8
    q_off, k_off, v_off = lead, lead + H * d, lead + H * d + G * d
    N = -(-(v_off + G * dv + 5) // 8) * 8
    proj = dev(rng.standard_normal((T, N)) * rng.uniform(0.2, 3.0, (T, 1)), dtype)
    qw, kw = dev(1 + 0.3 * rng.standard_normal(H * d)), dev(1 + 0.3 * rng.standard_normal(G * d))
    kc = torch.full((n_pages, G, page, d), 7.0, dtype=dtype, device="cuda")
    vc = torch.full((n_pages, G, page, dv), 7.0, dtype=dtype, device="cuda")
    q_out = torch.empty((T, H * d), dtype=dtype, device="cuda")
    x = host(proj)
    want_q = P.rms_norm(x[:, q_off:k_off], host(qw), 1e-4)
    want_k = P.rms_norm(x[:, k_off:v_off], host(kw), 1e-4).reshape(T, G, d)
    want_v = x[:, v_off:v_off + G * dv].reshape(T, G, dv)
    tol = dict(rtol=1e-2, atol=0.01) if dtype == BF16 else dict(rtol=0, atol=2e-5)
    args = (proj, q_off, k_off, v_off, qw, kw, 1e-4, q_out, kc, vc)
    ops.qk_row_norm_store(*args, None, H, G, d, dv, page)                        # queries alone
    np.testing.assert_allclose(host(q_out), want_q, **tol)
    assert float((kc - 7.0).abs().max()) == 0.0 and float((vc - 7.0).abs().max()) == 0.0
    ops.qk_row_norm_store(*args, st.slots[0], H, G, d, dv, page)
    touched = np.zeros((n_pages, page), dtype=bool)
    for t in range(T):
        pg, at = st.host_tables[st.host_seq[t], st.host_pos[t] // page], st.host_pos[t] % page
        touched[pg, at] = True
        np.testing.assert_allclose(host(kc[pg, :, at]), want_k[t], **tol)
        np.testing.assert_allclose(host(vc[pg, :, at]), want_v[t], rtol=0, atol=0)
    for c in (kc, vc):
        assert float((c.float().permute(0, 2, 1, 3)[~torch.from_numpy(touched).cuda()] - 7.0).abs().max()) == 0.0


def plain_rows(q, keys, vals, scale, st, H, G, gate, soft=P.softmax_plus_one):
    T = q.shape[0]
    out = np.zeros((T, H, vals[0].shape[-1]))
    for t in range(T):
        b, pos = st.host_seq[t], st.host_pos[t]
        for h in range(H):
            g = h // (H // G)
            out[t, h] = soft(keys[b][:pos + 1, g] @ q[t, h] * scale) @ vals[b][:pos + 1, g]
    return out * P.sigmoid(gate)


@pytest.mark.parametrize("dtype", [torch.float32, BF16])
@pytest.mark.parametrize("H,G,d,dv,page", [(4, 2, 32, 16, 8), (3, 3, 24, 8, 16), (1, 1, 8, 24, 16), (6, 2, 64, 32, 16),
                                           (2, 1, 128, 64, 8), (4, 4, 64, 128, 16), (8, 1, 64, 64, 32), (5, 5, 20, 12, 16)])
def test_attention_far_keys_under_one_in_the_denominator_and_a_gate_a_channel(dtype, H, G, d, dv, page):
    """Whole prompts, portions that start in the middle of a page, and single tokens in one launch.  Per head one key is made
    to carry the weight (query and key scaled): the first token, a page's last and first slot, a key far back, the token
    itself.  Elsewhere the scores are ordinary, and at a request's first tokens the one in the denominator takes about half."""
    from rust_llm_inference_server_b200 import ops
    rng = np.random.default_rng(H * 100 + d)
    ctx, qn = [333, 70, 129, 1, 2, 1100, 65, 150], [333, 1, 37, 1, 2, 1, 64, 1]
    n_pages = sum(-(-c // page) for c in ctx) + 3
    st = hand_step(ctx, qn, page, n_pages, rng)
    T = st.n_tokens
    keys, vals = [rng.standard_normal((c, G, d)) for c in ctx], [rng.standard_normal((c, G, dv)) for c in ctx]
    scale = 0.9 / np.sqrt(d)
    starts = np.concatenate([[0], np.cumsum(qn)])
    marked = [(int(starts[0] + qn[0] - 1), 0), (int(starts[5]), 5), (int(starts[2] + 20), 2), (int(starts[7]), 7), (int(starts[6] + 63), 6)]
    q = rng.standard_normal((T, H, d))
    for t, b in marked:
        pos = st.host_pos[t]
        far = [0, page - 1, page, 3 * page, pos // 2, pos - 1, pos]
        for h in range(H):
            j, g = min(max(far[h % len(far)], 0), pos), h // (H // G)
            q[t, h] = keys[b][j, g] * (9.0 / scale / float(keys[b][j, g] @ keys[b][j, g]))
    gate = dev(rng.standard_normal((T, H * dv + 11)) * 2, dtype)[:, 8:8 + H * dv]
    qd, out = dev(q.reshape(T, -1), dtype), torch.full((T, H * dv), float("nan"), dtype=dtype, device="cuda")
    kr, vr = [host(dev(k, dtype)) for k in keys], [host(dev(v, dtype)) for v in vals]
    kc, vc = fill_pools(st, kr, vr, page, n_pages, dtype)
    ops.launches_by_kernel.clear()
    ops.attention_biased(qd, kc, vc, out, None, gate, st, 0, H, G, d, dv, page, scale, 0, sinks=torch.zeros(H, device="cuda"))
    args = (host(qd).reshape(T, H, d), kr, vr, scale, st, H, G, host(gate).reshape(T, H, dv))
    want, got = plain_rows(*args), host(out).reshape(T, H, dv)
    err = np.abs(got - want).max(axis=(1, 2))
    assert np.isfinite(got).all() and err.max() <= (2e-5 if dtype == torch.float32 else 0.03), f"row {int(err.argmax())}: {err.max()}"
    plain = plain_rows(*args, soft=lambda s: np.exp(s - s.max()) / np.exp(s - s.max()).sum())
    assert np.abs(plain - want).max() > 0.2              # the test bites: a softmax without the one differs
    if dtype == BF16 and ops.biased_attention_takes_mma(dtype, H, G, d, dv):
        assert ops.launches_by_kernel.get("attention_bias.decode.mma.split") and ops.launches_by_kernel.get("attention_bias.prefill.mma")


@pytest.mark.parametrize("dtype", [torch.float32, BF16])
@pytest.mark.parametrize("T,W,I", [(3, 40, 24), (1, 128, 256), (16, 64, 100), (37, 100, 50), (150, 128, 256), (130, 64, 100), (300, 96, 384)])
def test_gated_unit_with_biases(dtype, T, W, I):
    """Through its products for few rows, for a few dozen and for many (the gating in the product's epilogue where the sizes
    allow), with the second bias added or left to the caller."""
    from rust_llm_inference_server_b200.parts.feed_forward import SwiGLU
    from rust_llm_inference_server_b200.parts.spec import SwiGLUSpec
    rng = np.random.default_rng(T + I)
    w = {n: dev(rng.standard_normal(s) / np.sqrt(s[1]), dtype) for n, s in (("g", (I, W)), ("u", (I, W)), ("d", (W, I)))}
    w.update({n: dev(rng.standard_normal(k)) for n, k in (("gb", I), ("ub", I), ("db", W))})
    ff = SwiGLU(SwiGLUSpec(W, I, "g", "u", "d", gate_bias="gb", up_bias="ub", down_bias="db"), dtype, "cuda")
    assert ff.tensors()["gb"] == (I,) and ff.tensors()["db"] == (W,)
    ff.load(SimpleNamespace(get=lambda name, role="matrix", share=False: w[name]))
    x = dev(rng.standard_normal((T, W)), dtype)
    st = SimpleNamespace(buffer=hand_step([1], [1], 8, 1, rng).buffer, n_tokens=T)
    xs = host(x)
    act = P.silu(xs @ host(w["g"]).T + host(w["gb"])) * (xs @ host(w["u"]).T + host(w["ub"]))
    act = to_bfloat16(act) if dtype == BF16 else act
    tol = dict(rtol=0, atol=3e-5 if dtype == torch.float32 else 0.06)
    np.testing.assert_allclose(host(ff.forward(x, st)), act @ host(w["d"]).T + host(w["db"]), **tol)
    np.testing.assert_allclose(host(ff.forward(x, st, defer_bias=True)), act @ host(w["d"]).T, **tol)


def test_dynamic_tanh_in_an_ordinary_block(model_root):
    """The norm under the pre-norm arrangement with one residual stream: another design's layer, built from specs."""
    from rust_llm_inference_server_b200.parts import DynamicTanhSpec, build_norm
    rng = np.random.default_rng(2)
    T, W = 6, 52
    for dtype in (torch.float32, BF16):
        n = build_norm(DynamicTanhSpec(W, "n", "n.b", "n.alpha"), dtype, "cuda")
        t = {"n": dev(rng.standard_normal(W)), "n.b": dev(rng.standard_normal(W)), "n.alpha": dev(0.6)}
        n.load(SimpleNamespace(get=lambda name, role="matrix", share=False: t[name]))
        st = SimpleNamespace(buffer=lambda name, shape, dt: torch.empty(shape, dtype=dt, device="cuda"))
        resid, delta = dev(rng.standard_normal((T, W))), dev(rng.standard_normal((T, W)), dtype)
        plain = {k: host(v) for k, v in t.items()}
        before = host(resid)
        tol = dict(rtol=1e-2 if dtype == BF16 else 0, atol=2e-5 if dtype == torch.float32 else 0.02)
        np.testing.assert_allclose(host(n.forward(resid, None, st)), P.dynamic_tanh(before, plain, "n"), **tol)
        rows = dev([4, 0], torch.int32)
        np.testing.assert_allclose(host(n.forward_rows(resid, delta, st, rows)), P.dynamic_tanh(before + host(delta), plain, "n")[[4, 0]], **tol)
        np.testing.assert_allclose(host(n.forward(resid, delta, st)), P.dynamic_tanh(before + host(delta), plain, "n"), **tol)
        np.testing.assert_allclose(host(resid), before + host(delta), rtol=0, atol=1e-6)


def test_streams_between_blocks_of_another_arrangement(model_root):
    """A hyper block between pre-norm blocks: it starts from their stream, and they go on from the sum of its streams."""
    from rust_llm_inference_server_b200.parts import HyperSpec, LayerSpec, RMSNormSpec, SwiGLUSpec, build_block
    from rust_llm_inference_server_b200.parts.base import Mixer, register_mixer
    rng = np.random.default_rng(3)
    T, W, S, eps = 5, 48, 3, 1e-5

    class Nothing(Mixer):
        def __init__(self, spec, dtype, device):
            pass

        def forward(self, x, step, cache, state, writes_cache=True):
            return x.clone()
    register_mixer("nothing", Nothing, replace=True)
    t = {n: dev(rng.standard_normal((64, W)) / 7) for n in ("g", "u")}
    t.update(d=dev(rng.standard_normal((W, 64)) / 8), read=dev(rng.standard_normal(S)), write=dev(rng.standard_normal(S)),
             mix=dev(rng.standard_normal((S, S)) / 2), n=dev(1 + 0.2 * rng.standard_normal(W)))
    src = SimpleNamespace(get=lambda name, role="matrix", share=False: t[name])
    norm, mixer, ff, hs = RMSNormSpec(W, eps, "n"), SimpleNamespace(kind="nothing"), SwiGLUSpec(W, 64, "g", "u", "d"), HyperSpec(S, "read", "write", "mix")
    blocks = [build_block(LayerSpec(norm, mixer, norm, ff, **k), torch.float32, "cuda")
              for k in ({}, dict(arrangement="hyper", hyper1=hs, hyper2=hs), {})]
    for b in blocks:
        for p in b.parts():
            p.load(src)
    bufs = {}
    st = SimpleNamespace(n_tokens=T, buffer=lambda name, shape, dt: bufs.setdefault((name, tuple(shape), dt), torch.empty(shape, dtype=dt, device="cuda")))
    x = rng.standard_normal((T, W))
    resid, pending = dev(x), None
    for b, nxt in zip(blocks, blocks[1:] + [None]):
        resid, pending = b.forward(resid, pending, st, None, None, next_block=nxt)
    got = host(resid) + host(pending)
    h = {k: host(v) for k, v in t.items()}
    nrm = lambda v: P.rms_norm(v, h["n"], eps)
    unit = lambda v: (P.silu(v @ h["g"].T) * (v @ h["u"].T)) @ h["d"].T

    def prenorm(v):
        v = v + nrm(v)
        return v + unit(nrm(v))
    x = prenorm(x)
    streams = np.stack([x] * S)
    for f in (lambda v: v, unit):
        streams = P.stream_update(streams, h["mix"], h["write"], f(nrm(P.stream_input(streams, h["read"]))))
    np.testing.assert_allclose(got, prenorm(streams.sum(axis=0)), rtol=0, atol=3e-4)


# ---- whole models ------------------------------------------------------------------------------

ALONE = {
    "attention_only": U.model(61, 48, 1e-5, 1.5, 2.0, 2, [U.attention(4, 2, 16, 8, 0.5)]),
    "delta_only": U.model(61, 48, 1e-5, 1.5, 2.0, 3, [U.channel_delta(4, 2, 8, 12, 4)]),
    "state_space_only": U.model(61, 48, 1e-5, 1.5, 2.0, 2, [U.mamba2(4, 12, 16, 2, 3, 4)]),
    "with_unit": U.model(61, 48, 1e-5, 1.0, 1.0, 4, [U.attention(2, 1, 24, 24, 0.3, 40)]),
    "looped": U.model(61, 48, 1e-5, 1.0, 1.0, 2, [U.channel_delta(2, 1, 12, 8, 2, 24), U.attention(2, 2, 8, 8, 0.6)], (0, 2, 3)),
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


@pytest.mark.parametrize("which", ["A", "D"])
def test_the_sum_of_the_streams_after_every_run_of_a_layer(model_root, which):
    d = U.make_dir(model_root, which)
    cfg, w = U.read_config(d), U.plain_weights(d)
    toks = requests_for(cfg, [45], seed=4)["r0"]
    want = P.forward(cfg, w, toks)[1]
    s = session(d, "float32", 64, 16)
    seen = []
    for blk in set(s.model.blocks):
        def tapped(*a, _inner=blk.forward, **k):
            r = _inner(*a, **k)
            seen.append(host(r[1].total()))
            return r
        blk.forward = tapped
    s.step({"step": 0, "entries": [{"id": "x", "tokens": toks, "want": [len(toks) - 1]}], "end": ["x"]})
    assert len(seen) == len(U.run_order(cfg))
    for i, (got, ref) in enumerate(zip(seen, want)):
        np.testing.assert_allclose(got, ref, rtol=0, atol=2e-4 * max(1.0, np.abs(ref).max() / 10), err_msg=f"after run {i}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which,page,lens", [("A", 16, [1, 50, 97, 200, 64, 17, 2]), ("A", 8, [130, 33, 2, 71, 40]),
                                             ("B", 16, [3, 150, 40, 2, 129, 1]), ("C", 16, [1, 70, 333, 2, 129, 64, 65]),
                                             ("D", 16, [90, 1, 33, 150, 2]), ("D", 32, [260, 31, 5, 90]),
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
        "mixed2": (R.mixed_trace(dict(reversed(list(reqs.items()))), seed=5, max_live=2), 2),   # two state slots for all
    }
    results = {}
    for fam, (steps, live) in families.items():
        s = session(d, dtype, R.live_token_peak(steps, max(64, page)), page, max_live=live)
        for pool in s.storage.pools:                         # whatever a page or a slot held before must not matter
            for t in (pool if isinstance(pool, tuple) else (pool,)):
                t.fill_(30.0)
        for state in s.storage.states:
            if state is not None:
                state.fill_(3.0)
        results[fam] = R.collect(s.step, steps)
        assert s.cache.check_invariants() == ""
        assert s.cache.num_free_pages(0) == s.cache.group(0).num_pages, fam
        assert s.cache.num_free_state_slots() == live, fam
        ok, what = ref.holds(results[fam])
        assert ok, f"{which} {dtype} {fam} vs plain: {what}"
    for fam in ("decode", "chunks", "mixed", "mixed2"):
        ok, what = ref.holds(results[fam], results["whole"], between=True)
        assert ok, f"{which} {dtype}: {fam} differs from whole by {what}"
    launched = ops.launches_by_kernel
    needed = {"stream_mix", "stream_mix.update", "stream_mix.update.rows", "qk_row_norm_store", "channel_delta.prepare",
              "channel_delta.scan", "state_space.prepare", "state_space.scan", "gate_group_norm", "head_norm_gate"}
    if dtype == "bfloat16":
        needed |= ({"stream_gemm.streams"} if U.CONFIGS[which]["width"] % 8 == 0 else set()) | ({"attention_bias.decode.mma", "attention_bias.prefill.mma"} if which in ("C", "E") else set())
        needed |= {"gemm_tcgen05.glu4"} if which == "E" else set()
    if max(lens) >= ops.GATED_DELTA_CHUNKS_FROM:
        needed |= {"channel_delta.chunks", "channel_delta.solve", "state_space.chunks"}
    assert needed <= set(launched), f"never launched {sorted(needed - set(launched))}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which,n,tail", [("A", 230, 215), ("B", 180, 170)])
def test_long_decoding(model_root, which, n, tail, dtype):
    d = U.make_dir(model_root, which)
    reqs = requests_for(U.CONFIGS[which], [n], seed=9)
    ref = plain_logits(d, reqs, dtype)
    steps = R.decode_trace(reqs, tail=tail)             # a page border every 8 tokens; steps replayed from a CUDA graph
    s = session(d, dtype, R.live_token_peak(steps), 8)
    ok, what = ref.holds(R.collect(s.step, steps))
    assert ok, what
    assert s.runner._graph_launches > 0


def plain_greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(np.argmax(P.forward(cfg, w, toks)[0][-1])))
    return toks[len(prompt):]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_entry_point(model_root, dtype):
    """Prompts of unequal length batched by the scheduler, portions of 16 tokens, decode steps from CUDA graphs and
    launched ahead; two seats, so the later prompts take over pages and state slots."""
    from rust_llm_inference_server_b200 import LLM, SamplingParams
    d = U.make_dir(model_root, "A")
    cfg, w = U.read_config(d), U.plain_weights(d)
    prompts = list(requests_for(cfg, [1, 9, 40, 23, 3], seed=12).values())
    llm = LLM(d, dtype=dtype, max_seq_len=128, num_blocks=40, block_size=8, max_num_seqs=2, max_batched_tokens=16)
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
    """random-weights and generate of the command line with a Papulix folder."""
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
    assert cfg["architecture"] == "Papulix" and set(w) == set(U.tensor_shapes(cfg))
    prompt = [5, 9, 200, 31, 7]
    r = rlis("generate", "--model", d, "--dtype", "f32", "--prompt-ids", ",".join(map(str, prompt)),
             "--max-tokens", "8", "--max-seq-len", "64", "--kv-cache-gb", "0.001", "--block-size", "8",
             "--max-num-seqs", "2")
    assert r.returncode == 0, r.stderr[-2000:]
    assert [int(t) for t in r.stdout.split()] == plain_greedy(cfg, w, prompt, 8)
