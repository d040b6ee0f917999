"""Papulix without a GPU: the configuration reader and what it refuses, the description against an independent list of
tensors, who keeps a cache and a state on which pass, the plain restatement against closed forms, and that the test
models' logits move far beyond the tolerances when a mechanism is left out."""

import copy

import numpy as np
import pytest

from tests import papulix_util as U
from tests.plain import papulix_plain as P


def test_reader_takes_every_size_and_constant_from_the_file():
    from rust_llm_inference_server_b200.config import ConfigError
    from rust_llm_inference_server_b200.config.papulix_config import PapulixConfig
    cfg = PapulixConfig.from_dict(U.CONFIGS["A"])
    assert (cfg.vocab, cfg.width, cfg.eps, cfg.embedding_scale, cfg.logit_scale, cfg.streams) == (211, 96, 1e-5, 2.0, 1.5, 3)
    assert cfg.run_order() == (0, 1, 2, 1, 2, 3, 4)
    m = cfg.layers[0].mixer
    assert (m.heads, m.vdim, m.state, m.groups, m.norm_groups, m.conv, m.inner, m.channels) == (6, 16, 24, 3, 2, 4, 96, 240)
    assert cfg.layers[0].ff == 40 and cfg.layers[1].ff is None
    a = cfg.layers[1].mixer
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale) == (4, 2, 16, 24, 0.5)
    c = cfg.layers[2].mixer
    assert (c.heads, c.kv_heads, c.dim, c.vdim, c.conv) == (4, 2, 16, 8, 3)
    assert PapulixConfig.from_dict(U.CONFIGS["B"]).run_order() == (0, 1, 2, 3, 4)

    def broken(edit):
        c = copy.deepcopy(U.CONFIGS["A"])
        edit(c)
        with pytest.raises(ConfigError):
            PapulixConfig.from_dict(c)
    broken(lambda c: c["layers"][1]["mixer"].update(heads=3))            # not a multiple of kv_heads
    broken(lambda c: c["layers"][2]["mixer"].update(kv_heads=3))
    broken(lambda c: c["layers"][0]["mixer"].update(groups=4))
    broken(lambda c: c["layers"][0]["mixer"].update(norm_groups=5))      # 96 channels in 5 parts
    broken(lambda c: c["layers"][0].update(type="mamba"))
    broken(lambda c: c["layers"][0]["mixer"].pop("state"))
    broken(lambda c: c["layers"][2]["mixer"].pop("conv"))
    broken(lambda c: c["layers"][1]["mixer"].pop("scale"))
    broken(lambda c: c["layers"][0]["mlp"].update(kind="moe"))
    broken(lambda c: c.pop("norm"))
    broken(lambda c: c.pop("streams"))
    broken(lambda c: c.update(streams=0))
    broken(lambda c: c["loop"].update(stop=6))
    broken(lambda c: c["loop"].update(start=4))
    broken(lambda c: c["loop"].pop("times"))


@pytest.mark.parametrize("which", sorted(U.CONFIGS))
def test_description_lists_the_tensors_and_the_runs(which):
    from rust_llm_inference_server_b200.models.model import build_model
    cfg = U.CONFIGS[which]
    model = build_model(cfg, "float32", "cpu")
    want = U.tensor_shapes(cfg, (None, None))                            # the ranks are the checkpoint's
    got = model.tensors()
    assert set(got) == set(want)
    for name, shape in got.items():
        assert tuple(shape) == tuple(want[name]), name
    order = U.run_order(cfg)
    assert [c.layer for c in model.calls] == order and [c.cache for c in model.calls] == list(range(len(order)))
    for run, i in enumerate(order):                                      # every pass has a cache or state of its own
        m = cfg["layers"][i]["mixer"]
        cache = model.cache_slot_specs[run] if run < len(model.cache_slot_specs) else None
        state = model.call_state_specs[run]
        if cfg["layers"][i]["type"] == "attention":
            assert state is None
            assert (cache.n_kv_heads, cache.head_dim, cache.v_head_dim or cache.head_dim, cache.window or None) == \
                (m["kv_heads"], m["dim"], m["vdim"], None)
        else:
            qk = m["groups"] * m["state"] if "state" in m else m["kv_heads"] * m["dim"]
            floats = m["heads"] * m["vdim"] * m.get("state", m.get("dim")) + (m["conv"] - 1) * (2 * qk + m["heads"] * m["vdim"])
            assert cache is None and tuple(state.shape) == (-(-floats // 4) * 4,)
    assert model.graph_safe


def test_checkpoints_are_checked_as_a_whole(tmp_path):
    from rust_llm_inference_server_b200.models.model import build_model
    from rust_llm_inference_server_b200.weights.loader import WeightError
    from rust_llm_inference_server_b200.weights.safetensors_io import open_model_dir
    import torch
    cfg = U.CONFIGS["A"]

    def load(which, edit):
        d = U.make_dir(str(tmp_path), which, cfg, 1, edit)
        build_model(cfg, "float32", "cpu").load(open_model_dir(d))
    load("fine", lambda w: None)
    # what a layer without a feed-forward does not read may be there
    load("more", lambda w: w.update({"l1.norm2": torch.ones(96), "l1.hc2.in": torch.ones(3)}))
    for name, edit in (("missing", lambda w: w.pop("l2.hc1.mix")), ("extra", lambda w: w.update({"l0.mix.q": torch.ones(3)})),
                       ("shape", lambda w: w.update({"l2.mix.dt_bias": torch.ones(4)}))):
        with pytest.raises(WeightError):
            load(name, edit)
    with pytest.raises(ValueError):                                      # two ranks for one low-rank map
        load("ranks", lambda w: w.update({"l2.mix.a1": torch.ones(9, 96)}))


def test_random_weights_mode_knows_the_design():
    from rust_llm_inference_server_b200.weights.random_init import random_tensors
    cfg = U.CONFIGS["D"]
    w = random_tensors(cfg, 4)
    m = cfg["layers"][1]["mixer"]
    want = U.tensor_shapes(cfg, (m["dim"], m["vdim"]))
    assert {k: tuple(v.shape) for k, v in w.items()} == {k: tuple(v) for k, v in want.items()}
    assert abs(float(np.diag(w["l0.hc1.mix"].float().numpy()).mean()) - 1.0) < 0.3


def test_plain_mechanisms_against_closed_forms():
    rng = np.random.default_rng(0)
    # a short convolution reads the last taps - 1 inputs and zeros before the start
    x, taps = rng.standard_normal((5, 2)), rng.standard_normal((2, 3))
    y = P.short_conv(x, taps)
    assert np.allclose(y[0], P.silu(taps[:, 2] * x[0])) and np.allclose(y[3], P.silu((taps.T * x[1:4]).sum(axis=0)))
    assert np.allclose(P.short_conv(x, taps, np.ones(2))[0], P.silu(taps[:, 2] * x[0] + 1.0))
    # the delta rule with beta 1, no decay and orthonormal keys stores values exactly
    k, v = np.eye(3), rng.standard_normal((3, 2))
    o = P.channel_decay_delta(np.eye(3)[[0, 0, 1]], k, v, np.ones(3), np.ones((3, 3)))
    assert np.allclose(o, [v[0], v[0], v[1]])
    # a decay acts on the rows that belong to its key channel, before the write
    g = np.array([[1.0, 1.0, 1.0], [0.5, 1.0, 1.0], [0.5, 0.25, 1.0]])
    o = P.channel_decay_delta(np.eye(3)[[0, 0, 1]], k, v, np.ones(3), g)
    assert np.allclose(o, [v[0], 0.5 * v[0], 0.25 * v[1]])
    # beta 0 writes nothing; a second write along a key replaces its value
    o = P.channel_decay_delta(np.eye(3)[[0, 0, 0]], k[[0, 0, 0]], v, np.array([1.0, 0.0, 1.0]), np.ones((3, 3)))
    assert np.allclose(o, [v[0], v[0], v[2]])
    # state space: y_t = sum_j exp(log_a (dt_(j+1) + .. + dt_t)) dt_j (C_t . B_j) x_j + D x_t
    T = 6
    xs, B, C, dt = rng.standard_normal((T, 3)), rng.standard_normal((T, 2)), rng.standard_normal((T, 2)), rng.uniform(0.1, 1, T)
    got = P.state_space(xs, B, C, dt, -0.7, 1.3)
    for t in range(T):
        want = sum(np.exp(-0.7 * dt[j + 1:t + 1].sum()) * dt[j] * (C[t] @ B[j]) * xs[j] for j in range(t + 1)) + 1.3 * xs[t]
        assert np.allclose(got[t], want)
    # gate before norm, each part by its own root mean square
    y, z = rng.standard_normal((2, 4)), rng.standard_normal((2, 4))
    got = P.gated_group_norm(y, z, np.array([1.0, 2.0, 1.0, 1.0]), 2, 0.0)
    a = y * P.silu(z)
    assert np.allclose(got[:, 1], 2 * a[:, 1] / np.sqrt((a[:, :2] ** 2).mean(axis=1))) and np.allclose(np.abs(got[:, 2:]).max(), np.abs(got[:, 2:]).max())
    assert np.allclose((got[:, 2:] ** 2).mean(axis=1), 1.0)
    # the softmax with one added, also for large scores
    assert np.allclose(P.softmax_plus_one(np.array([0.0])), [0.5])
    assert np.allclose(P.softmax_plus_one(np.array([-800.0, 800.0])), [0.0, 1.0])
    p = P.softmax_plus_one(np.array([0.3, -1.0]))
    assert np.allclose(p, np.exp([0.3, -1.0]) / (1 + np.exp([0.3, -1.0]).sum()))
    # streams: every new one from the old ones; rows of the matrix are sources, columns targets
    st = rng.standard_normal((2, 1, 3))
    mix, out, y = np.array([[0.5, 2.0], [3.0, 0.1]]), np.array([1.0, -1.0]), rng.standard_normal((1, 3))
    new = P.stream_update(st, mix, out, y)
    assert np.allclose(new[0], 0.5 * st[0] + 3.0 * st[1] + y) and np.allclose(new[1], 2.0 * st[0] + 0.1 * st[1] - y)
    assert np.allclose(P.stream_input(st, np.array([2.0, -1.0])), 2 * st[0] - st[1])


@pytest.mark.parametrize("which", ["A", "D"])
def test_every_mechanism_counts_in_the_test_models(which):
    """The logits of the test models move far beyond the tolerances when a mechanism is left out or read otherwise."""
    import torch
    cfg = U.CONFIGS[which]
    w = {k: v.to(torch.float64).numpy() for k, v in U.draw_weights(cfg, U.SEEDS[which], U.RANKS[which]).items()}
    toks = np.random.default_rng(1).integers(0, cfg["vocab"], size=60).tolist()
    base = P.forward(cfg, w, toks)[0]

    def moved(cfg2=None, w2=None, least=0.02):
        got = P.forward(cfg2 or cfg, w2 or w, toks)[0]
        d = (got - base)[20:]
        assert np.sqrt((d * d).mean()) / base.std() > least

    def edited(fn):
        c = copy.deepcopy(cfg)
        fn(c)
        return c

    def replaced(name, value):
        assert name in w, name
        return {**w, name: value(w[name])}
    at = {l["type"]: i for i, l in reversed(list(enumerate(cfg["layers"])))}
    dense = next(i for i, l in enumerate(cfg["layers"]) if l["mlp"])
    zero, one = np.zeros_like, np.ones_like
    moved(edited(lambda c: c["loop"].update(times=c["loop"]["times"] - 1)))
    moved(edited(lambda c: c["embedding"].update(scale=c["embedding"]["scale"] * 1.5)))
    moved(edited(lambda c: c.update(logit_scale=c["logit_scale"] * 1.5)))
    a = f"l{at['attention']}.mix."
    moved(edited(lambda c: c["layers"][at["attention"]]["mixer"].update(scale=0.0)))
    for name in ("q.norm", "k.norm"):
        moved(w2=replaced(a + name, one), least=0.005)
    moved(w2=replaced(a + "g", zero))
    c = f"l{at['channel_delta']}.mix."
    for name in ("b", "a2", "g2", "dt_bias", "A_log"):
        moved(w2=replaced(c + name, zero), least=0.005)
    for name in ("q.conv", "k.conv", "v.conv"):                          # only the current token's tap
        moved(w2=replaced(c + name, lambda x: np.where(np.arange(x.shape[1]) < x.shape[1] - 1, 0.0, x)))
    moved(w2=replaced(c + "norm", one), least=0.005)
    s = f"l{at['mamba2']}.mix."
    for name in ("conv.b", "dt_bias", "A_log", "D"):
        moved(w2=replaced(s + name, zero), least=0.01)
    moved(w2=replaced(s + "norm", one), least=0.005)
    for name in ("mlp.gate.b", "mlp.up.b", "mlp.down.b", "norm1.b", "norm2.b"):
        moved(w2=replaced(f"l{dense}." + name, zero), least=0.005)
    moved(w2=replaced(f"l{dense}.norm1.alpha", lambda x: x * 1.5))
    moved(w2=replaced("final.norm.b", zero))
    for name in ("hc1.in", "hc1.out", "hc2.in", "hc2.out"):
        moved(w2=replaced(f"l{dense}." + name, one), least=0.005)
    for name in ("hc1.mix", "hc2.mix"):
        moved(w2=replaced(f"l{dense}." + name, np.transpose), least=0.01)
    # a softmax without the one in the denominator
    import unittest.mock as mock
    with mock.patch.object(P, "softmax_plus_one", lambda s: np.exp(s - s.max()) / np.exp(s - s.max()).sum()):
        moved(least=0.01)
