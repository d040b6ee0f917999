"""Dotivik without a GPU: the configuration reader and what it refuses, the description against an independent list of
tensors, which calls keep which cache and where a pass starts, the plain restatement against closed forms, and that the test
models' logits move far beyond the tolerances when a mechanism is left out."""

import copy
import unittest.mock as mock

import numpy as np
import pytest

from tests import dotivik_util as U
from tests.plain import dotivik_plain as P


def test_reader_takes_every_size_and_constant_from_the_file():
    from rust_llm_inference_server_b200.config import ConfigError
    from rust_llm_inference_server_b200.config.dotivik_config import DotivikConfig
    cfg = DotivikConfig.from_dict(U.CONFIGS["A"])
    assert (cfg.vocab, cfg.width, cfg.eps) == (211, 96, 1e-5)
    assert cfg.runs() == ((0, False), (1, True), (2, False), (1, True), (2, False), (3, False))
    m = cfg.layers[0].mixer
    assert (m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank, m.scale, m.window, m.rot.dims, m.rot.base) == \
        (3, 16, 8, 24, 40, 0.3, 7, 8, 10000.0)
    assert cfg.layers[0].ff == 40 and cfg.layers[1].ff is None
    a = cfg.layers[1].mixer
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.softcap, a.diff, a.rot.dims, a.rot.base) == \
        (4, 2, 16, 24, 0.5, 6.0, 0.4, 8, 500.0)
    assert DotivikConfig.from_dict(U.CONFIGS["D"]).runs() == ((0, False), (1, False))
    never = copy.deepcopy(U.CONFIGS["A"])
    never["loop"]["times"] = 0
    assert DotivikConfig.from_dict(never).runs() == ((0, False), (3, False))

    def broken(edit):
        c = copy.deepcopy(U.CONFIGS["A"])
        edit(c)
        with pytest.raises(ConfigError):
            DotivikConfig.from_dict(c)
    broken(lambda c: c["layers"][1]["mixer"].update(heads=3))            # not a multiple of kv_heads
    broken(lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7))
    broken(lambda c: c["layers"][1]["mixer"]["rot"].update(dims=18))     # more than a map has
    broken(lambda c: c["layers"][1]["mixer"].update(softcap=0.0))
    broken(lambda c: c["layers"][1]["mixer"].pop("diff"))
    broken(lambda c: c["layers"][1]["mixer"].pop("scale"))
    broken(lambda c: c["layers"][0]["mixer"]["rot"].update(dims=6))      # the whole shared part turns
    broken(lambda c: c["layers"][0]["mixer"].pop("mask"))
    broken(lambda c: c["layers"][0]["mixer"]["mask"].update(size=0))
    broken(lambda c: c["layers"][0]["mixer"].pop("kv_rank"))
    broken(lambda c: c["layers"][0].update(type="latent"))
    broken(lambda c: c["layers"][0]["mlp"].update(kind="moe"))
    broken(lambda c: c.pop("norm"))
    broken(lambda c: c["loop"].update(stop=5))
    broken(lambda c: c["loop"].update(start=4))
    broken(lambda c: c["loop"].pop("times"))


@pytest.mark.parametrize("which", sorted(U.CONFIGS))
def test_description_lists_the_tensors_and_the_runs(which):
    from rust_llm_inference_server_b200.models.model import build_model
    from rust_llm_inference_server_b200.parts.block import ParallelBlock, StreamJoin
    cfg = U.CONFIGS[which]
    model = build_model(cfg, "float32", "cpu")
    want = U.tensor_shapes(cfg)
    got = model.tensors()
    assert {k: tuple(v) for k, v in got.items()} == {k: tuple(v) for k, v in want.items()}
    order = U.runs(cfg)
    assert [c.layer for c in model.calls] == order and [c.cache for c in model.calls] == list(range(len(order)))
    for run, i in enumerate(order):                                      # every pass has a cache of its own
        m, spec = cfg["layers"][i]["mixer"], model.cache_slot_specs[run]
        assert model.call_state_specs[run] is None
        if cfg["layers"][i]["type"] == "attention":
            assert (spec.n_kv_heads, spec.head_dim, spec.v_head_dim or spec.head_dim, spec.window or None, spec.values) == \
                (m["kv_heads"], 2 * m["dim"], m["vdim"], None, True)
        else:
            assert (spec.n_kv_heads, spec.head_dim, spec.window, spec.values) == (1, m["kv_rank"] + m["rot_dim"], m["mask"]["size"], False)
    starts = [] if cfg.get("loop") is None else [r for r, i in enumerate(order) if i == cfg["loop"]["start"]]
    assert [r for r, c in enumerate(model.calls) if c.entry is not None] == starts
    stations = [b for b, _ in model._stations]
    assert len(stations) == len(order) + len(starts) and all(isinstance(b, (ParallelBlock, StreamJoin)) for b in stations)
    assert len({id(b) for b in stations if isinstance(b, StreamJoin)}) == min(1, len(starts))      # one map for all passes
    assert model.graph_safe


def test_checkpoints_are_checked_as_a_whole(tmp_path):
    from rust_llm_inference_server_b200.models.model import build_model
    from rust_llm_inference_server_b200.weights.loader import WeightError
    from rust_llm_inference_server_b200.weights.safetensors_io import open_model_dir
    import torch

    def load(which, edit, name="A", dtype="float32"):
        model = build_model(U.CONFIGS[name], dtype, "cpu")
        model.load(open_model_dir(U.make_dir(str(tmp_path), which, U.CONFIGS[name], 1, edit)))
        return model
    load("fine", lambda w: None)
    load("more", lambda w: w.update({"loop.in": torch.ones(100, 200)}), "D")     # a map that no pass reads may be there
    for name, edit in (("missing", lambda w: w.pop("loop.in")), ("extra", lambda w: w.update({"l0.mix.k": torch.ones(3)})),
                       ("shape", lambda w: w.update({"l1.mix.lq2": torch.ones(4)}))):
        with pytest.raises(WeightError):
            load(name, edit)
    # the matrices that read a block's normed input are one, and the parts keep views of it
    m = load("fine_c", lambda w: None, "C", "bfloat16")
    for b, layer in zip(m.blocks, U.CONFIGS["C"]["layers"]):
        n = b.joint.n_plain
        assert n % 8 == 0 and b.joint.w.shape == (n + 2 * layer["mlp"]["ff"], 128)
        assert b.mixer.w_in.data_ptr() == b.joint.w.data_ptr() and b.feed_forward.w_gate_up.data_ptr() == b.joint.w[n:].data_ptr()
    w = U.plain_weights(U.make_dir(str(tmp_path), "fine_c"))
    assert abs(m.blocks[2].mixer.lam - P.head_weight(w, "l2.mix.", 0.6)) < 1e-6


def test_random_weights_mode_knows_the_design():
    from rust_llm_inference_server_b200.weights.random_init import random_tensors
    for which in ("A", "D"):
        w = random_tensors(U.CONFIGS[which], 4)
        assert {k: tuple(v.shape) for k, v in w.items()} == {k: tuple(v) for k, v in U.tensor_shapes(U.CONFIGS[which]).items()}
    assert abs(float(w["l0.norm1"].float().mean()) - 1.0) < 0.05


def test_a_layer_norm_is_not_taken_for_an_rms_norm():
    from rust_llm_inference_server_b200.parts import LayerNormSpec, LayerSpec, NoPositionSpec, build_block
    from rust_llm_inference_server_b200.parts.spec import GQAAttentionSpec
    norm = LayerNormSpec(32, 1e-5, "n")
    mixer = GQAAttentionSpec(32, 2, 1, 16, "q", "k", "v", "o", NoPositionSpec())
    for arrangement in ("sandwich", "outnorm", "postnorm", "hyper"):
        with pytest.raises((ValueError, AttributeError)):
            build_block(LayerSpec(norm, mixer, None, None, arrangement=arrangement, post_norm1=norm), "float32", "cpu")
    with pytest.raises(ValueError):                      # sublayers side by side have one norm
        build_block(LayerSpec(norm, mixer, norm, None, arrangement="parallel"), "float32", "cpu")


def test_plain_mechanisms_against_closed_forms():
    rng = np.random.default_rng(0)
    # a layer norm has no mean and unit variance, and a shift of the row changes nothing
    x = rng.standard_normal((3, 40)) * 2 + 5
    y = P.layer_norm(x, 1.0, 0.0)
    assert np.allclose(y.mean(axis=1), 0) and np.allclose((y * y).mean(axis=1), 1) and np.allclose(P.layer_norm(x + 9.0, 1.0, 0.0), y)
    # rotations keep lengths, leave the rest alone, and make scores depend on distances
    rot = {"dims": 6, "base": 50.0}
    for turn, partner in ((P.rotate_neighbours, lambda i: i ^ 1), (P.rotate_halves, lambda i: (i + 3) % 6)):
        v = rng.standard_normal((1, 1, 10))
        r = turn(np.repeat(v, 30, axis=0), rot)
        assert np.allclose(r[0], v[0]) and np.allclose(r[..., 6:], v[..., 6:])
        assert np.allclose((r * r).sum(axis=-1), (v * v).sum())
        s = r[:, 0] @ r[:, 0].T
        assert np.allclose(s[4, 1], s[20, 17]) and np.allclose(s[9, 2], s[27, 20])
        one = np.zeros((2, 1, 10))
        one[:, 0, 1] = 1.0
        got = turn(one, rot)[1, 0]
        f = 50.0 ** (-2.0 * (0 if turn is P.rotate_neighbours else 1) / 6)
        assert np.isclose(got[1], np.cos(f)) and np.isclose(abs(got[partner(1)]), abs(np.sin(f)))
    # a capped score stays below the cap and starts with slope one
    assert np.isclose(P.capped(1e-4, 3.0), 1e-4) and np.isclose(P.capped(1e3, 3.0), 3.0) and P.capped(-50.0, 3.0) > -3.0001
    # windows: itself and the ones before it
    v = np.eye(5)
    got = P.softmax_attention(np.zeros((5, 2)), np.zeros((5, 2)), v, lambda r: r, 2)
    assert np.allclose(got[0], v[0]) and np.allclose(got[3], (v[2] + v[3]) / 2)
    assert np.allclose(P.softmax_attention(np.zeros((5, 2)), np.zeros((5, 2)), v, lambda r: r)[3], v[:4].mean(axis=0))
    # the difference of two maps, normed a head
    a1, a2 = rng.standard_normal((2, 4, 6))
    got = P.difference_of_maps(a1, a2, 0.7, 0.4, 0.0)
    assert np.allclose((got * got).mean(axis=1), 0.36) and np.allclose(got[:, 0] / got[:, 1], (a1 - 0.7 * a2)[:, 0] / (a1 - 0.7 * a2)[:, 1])
    z = {"lq1": np.array([1.0, 0.0]), "lk1": np.array([np.log(3.0), 5.0]), "lq2": np.zeros(2), "lk2": np.ones(2)}
    assert np.isclose(P.head_weight(z, "", 0.25), 3.0 - 1.0 + 0.25)
    # gelu's tanh form as a gate with a cubic argument
    from rust_llm_inference_server_b200.parts.spec import GELU_TANH
    g = np.linspace(-6, 6, 101)
    assert np.allclose(P.gelu_tanh(g), g * P.sigmoid(GELU_TANH["slope"] * (g + GELU_TANH["cubic"] * g ** 3)), atol=1e-12)
    # the map in front of a pass reads the stream first, then the embedding
    w = np.concatenate([2 * np.eye(3), 5 * np.eye(3)], axis=1)
    assert np.allclose(P.pass_input(np.array([[1.0, 2, 3]]), np.array([[10.0, 0, 1]]), w), [[52.0, 4, 11]])


@pytest.mark.parametrize("which", ["A", "C"])
def test_every_mechanism_counts_in_the_test_models(which):
    """The logits of the test models move far beyond the tolerances when a mechanism is left out or read otherwise."""
    import torch
    cfg = U.CONFIGS[which]
    w = {k: v.to(torch.float64).numpy() for k, v in U.draw_weights(cfg, U.SEEDS[which]).items()}
    toks = np.random.default_rng(1).integers(0, cfg["vocab"], size=120).tolist()
    base = P.forward(cfg, w, toks)[0]

    def moved(cfg2=None, w2=None, least=0.03, **patches):
        with mock.patch.multiple(P, **patches) if patches else mock.patch.object(P, "kept", P.kept):
            got = P.forward(cfg2 or cfg, w2 or w, toks)[0]
        d = (got - base)[105:]
        assert np.sqrt((d * d).mean()) / base.std() > least

    def edited(fn):
        c = copy.deepcopy(cfg)
        fn(c)
        return c
    at = {l["type"]: i for i, l in reversed(list(enumerate(cfg["layers"])))}
    mixer = lambda c, kind: c["layers"][at[kind]]["mixer"]
    moved(edited(lambda c: c["loop"].update(times=c["loop"]["times"] - 1)))
    moved(edited(lambda c: mixer(c, "attention").update(softcap=1e6)), least=0.005)
    moved(edited(lambda c: mixer(c, "attention").update(diff=0.9)), least=0.02)
    moved(edited(lambda c: mixer(c, "attention").update(scale=0.0)))
    moved(edited(lambda c: mixer(c, "attention")["rot"].update(dims=mixer(c, "attention")["rot"]["dims"] - 4)), least=0.01)
    moved(edited(lambda c: mixer(c, "latent_attention").update(scale=0.0)))
    for step in (-1, 1):
        moved(edited(lambda c: mixer(c, "latent_attention")["mask"].update(size=mixer(c, "latent_attention")["mask"]["size"] + step)), least=0.002)
    moved(edited(lambda c: mixer(c, "latent_attention")["rot"].update(base=2.0)))
    a, l = f"l{at['attention']}.mix.", f"l{at['latent_attention']}.mix."
    for name in (a + "g", l + "g", a + "lq1", a + "lk2"):
        moved(w2={**w, name: np.zeros_like(w[name])}, least=0.002 if "lq" in name or "lk" in name else 0.03)
    moved(w2={**w, l + "dkv.norm": np.ones_like(w[l + "dkv.norm"])}, least=0.01)
    moved(w2={**w, "final.norm": np.ones_like(w["final.norm"])})
    W = cfg["width"]
    moved(w2={**w, "loop.in": np.concatenate([w["loop.in"][:, W:], w["loop.in"][:, :W]], axis=1)})
    moved(layer_norm=lambda x, weight, eps: P.rms_norm(x, weight, eps))
    moved(rotate_neighbours=P.rotate_halves)
    moved(rotate_halves=P.rotate_neighbours)
    moved(difference_of_maps=lambda a1, a2, lam, diff, eps: (a1 - lam * a2) * (1 - diff))
    moved(gelu_tanh=lambda z: z * P.sigmoid(z), least=0.02)
