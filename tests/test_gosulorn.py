"""Gosulorn without a GPU: the configuration reader and its errors, the tensor names and shapes of every test configuration,
which layer runs with whose tensors and what every run keeps, caches of several memories, and the plain mechanisms on
cases worked out by hand."""
import copy
import math

import numpy as np
import pytest
import torch

import plain_gosulorn as P
from gosulorn_configs import CONFIGS, make_weights, ranks_of, tensor_shapes, write_model_dir


def _spec(cfg):
    from kappai_b200.config.registry import config_from_dict
    arch, c = config_from_dict(cfg)
    assert arch.name == "Gosulorn"
    return arch.build_spec(c)


def _model(cfg):
    from kappai_b200.engine.model import Model
    from kappai_b200.parts.base import BuildEnv
    return Model(_spec(cfg), BuildEnv(torch.device("cpu"), torch.float32, 32))


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_tensor_names_and_shapes(name):
    cfg = CONFIGS[name][0]
    table, want = _model(cfg).weight_table(), tensor_shapes(cfg)
    assert set(table) == set(want)
    for n, ws in table.items():
        assert ws.fits(want[n]), (n, ws.shape, want[n])
        assert not ws.fits(want[n] + (1,)) and not ws.fits(tuple(x + 1 for x in want[n]))


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_layer_runs_and_what_every_run_keeps(name):
    from kappai_b200.cache import PagedKVSpec, StateSpec, leaf_specs
    cfg = CONFIGS[name][0]
    m = _model(cfg)
    assert len(m.schedule) == len(cfg["layers"]) and len(m.blocks) == sum(l.get("weights_of") is None for l in cfg["layers"])
    for i, layer in enumerate(cfg["layers"]):
        j = layer.get("weights_of")
        if j is not None:
            assert m.schedule[i].layer == m.schedule[j].layer and m.schedule[i].cache_of is None       # same tensors, a memory of its own
    conv = lambda x: (x["conv"] - 1) * (2 * x["kv_heads"] * x["dim"] + x["heads"] * x["vdim"])
    for layer, spec in zip(cfg["layers"], m.cache_specs()):
        mix, leaves = layer["mixer"], list(leaf_specs(spec))
        if layer["type"] == "gla":
            assert leaves == [StateSpec((mix["heads"] * mix["dim"] * mix["vdim"],), "float32")]
        elif layer["type"] == "delta":
            assert leaves == [StateSpec((mix["heads"] * mix["dim"] * mix["vdim"] + conv(mix),), "float32")]
        else:
            left, right = mix["left"], mix["right"]
            assert isinstance(leaves[0], PagedKVSpec) and leaves[0].num_kv_heads == left["kv_heads"]
            assert leaves[0].window == (left.get("mask") or {}).get("size") and leaves[0].head_dim >= max(left["dim"], left["vdim"])
            assert leaves[-1] == StateSpec((right["heads"] * right["dim"] * right["vdim"] + conv(right),), "float32")
            assert len(leaves) == (3 if left["conv"] > 1 else 2)
            if left["conv"] > 1:
                assert leaves[1].shape[0] == (left["conv"] - 1) * (left["heads"] + 2 * left["kv_heads"]) * leaves[0].head_dim


def test_parts_and_their_constants_come_from_the_configuration():
    cfg = CONFIGS["A"][0]
    m = _model(cfg)
    par, delta, gla = (b.mixer for b in m.blocks)
    left, right = par.mixers["left"], par.mixers["right"]
    assert left.window == 20 and left.scale == 0.35 and left.taps == 3 and left.out_scale == 1.3 and left.bias and left.exact_weights
    assert left.position.scaling == (4.0,) and left.position.rotary_dim == 8 and left.position.theta == 1000.0
    assert right.out_scale == 0.6 and right.per_channel and right.gate == "sigmoid" and right.gate_rank == "low" and right.taps == 4
    assert not delta.per_channel and delta.gate == "silu" and delta.gate_rank == "full" and (delta.H, delta.G) == (6, 3)
    assert gla.tau == 4.0 and delta.eps == gla.eps == cfg["norm"]["eps"]
    assert m.residual.S == 3 and m.head.tied and m.graph_safe
    assert all(b.ffn.activation == "gelu_tanh" for b in m.blocks)
    b = _model(CONFIGS["B"][0])
    assert b.blocks[0].ffn is None and b.blocks[0].sublayers == 1 and b.blocks[1].mixer.mixers["left"].window is None
    assert b.blocks[1].mixer.mixers["left"].position.fused_rotary()[2] == 0


@pytest.mark.parametrize("change,word", [
    (lambda c: c.pop("vocab"), "vocab"),
    (lambda c: c.pop("streams"), "streams"),
    (lambda c: c.update(streams=0), "streams"),
    (lambda c: c["norm"].pop("eps"), "norm.eps"),
    (lambda c: c["layers"][0].update(type="conv"), "type"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=4), "kv_heads"),
    (lambda c: c["layers"][1]["mixer"].pop("conv"), "conv"),
    (lambda c: c["layers"][2]["mixer"].pop("tau"), "tau"),
    (lambda c: c["layers"][2]["mixer"].update(tau=0), "tau"),
    (lambda c: c["layers"][0]["mixer"].pop("left_scale"), "left_scale"),
    (lambda c: c["layers"][0]["mixer"].pop("right"), "right"),
    (lambda c: c["layers"][0]["mixer"]["left"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=7), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=18), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"]["scaling"].update(factor=0), "factor"),
    (lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(size=0), "mask.size"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "kind"),
    (lambda c: c["layers"][3].update(weights_of=3), "weights_of"),
    (lambda c: c["layers"][3].update(weights_of=9), "weights_of"),
    (lambda c: c["layers"][3].update(weights_of=0), "type"),
    (lambda c: c["layers"][3]["mixer"].update(heads=3), "mixer"),
])
def test_configuration_errors_name_the_key(change, word):
    from kappai_b200.config.schema import ConfigError
    cfg = copy.deepcopy(CONFIGS["A"][0])
    change(cfg)
    with pytest.raises(ConfigError) as e:
        _spec(cfg)
    assert word in str(e.value)


def test_loading_checks_shapes_and_ranks_come_from_the_file(tmp_path):
    from kappai_b200.config.schema import ConfigError
    from kappai_b200.weights.loader import WeightError, load_weights
    cfg, seed = CONFIGS["A"]
    w = make_weights(cfg, seed)
    m = _model(cfg)
    load_weights(m, write_model_dir(cfg, w, str(tmp_path / "a")))
    ra, rg = ranks_of(cfg)
    right = m.blocks[0].mixer.mixers["right"]
    assert right.w_decay.shape[1] >= ra and right.w_gate.shape[1] >= rg
    assert torch.equal(right.w_decay[:, :ra], w["l0.mix.right.a2"].float()) and not right.w_decay[:, ra:].any()
    with pytest.raises(WeightError) as e:
        load_weights(_model(cfg), write_model_dir(cfg, dict(w, **{"l1.mix.q": w["l1.mix.q"][:-1]}), str(tmp_path / "b")))
    assert "l1.mix.q" in str(e.value)
    with pytest.raises(ConfigError):
        load_weights(_model(cfg), write_model_dir(cfg, dict(w, **{"l2.mix.a2": w["l2.mix.a2"][:, :-1]}), str(tmp_path / "c")))
    # the norm and coefficients of a feed-forward that a layer does not have may be there unread
    cb, sb = CONFIGS["B"]
    wb = make_weights(cb, sb)
    extra = {"l0.norm2": torch.ones(48).bfloat16(), "l0.hc2.in": torch.ones(2).bfloat16(), "l0.hc2.out": torch.ones(2).bfloat16(),
             "l0.hc2.mix": torch.eye(2).bfloat16()}
    load_weights(_model(cb), write_model_dir(cb, dict(wb, **extra), str(tmp_path / "d")))


def test_caches_of_several_memories():
    from kappai_b200.cache.spec import CompositeSpec, PagedKVSpec, StateSpec, leaf_specs
    from kappai_b200.cache.storage import CacheStorage, CompositeView, KVLayerView, StateView
    kv = PagedKVSpec(2, 16, 20)
    both = CompositeSpec((CompositeSpec((kv, StateSpec((6,)))), StateSpec((2, 3))))
    assert [type(s).__name__ for s in leaf_specs(both)] == ["PagedKVSpec", "StateSpec", "StateSpec"] and list(leaf_specs(None)) == []
    st = CacheStorage([both, kv, None, both, StateSpec((4,))], [None, None, None, 0, None], {kv.group_key: 3}, 8, 2, torch.float32,
                      torch.device("cpu"))
    v = st.views[0]
    assert isinstance(v, CompositeView) and isinstance(v.parts[0], CompositeView)
    assert isinstance(v.parts[0].parts[0], KVLayerView) and isinstance(v.parts[0].parts[1], StateView) and v.parts[1].tensor.shape == (2, 2, 3)
    pool = st.pools[kv.group_key]
    assert pool.shape[0] == 2 and v.parts[0].parts[0].tensor.data_ptr() == pool[0].data_ptr() and st.views[1].tensor.data_ptr() == pool[1].data_ptr()
    lent = st.views[3]                                           # a borrower sees the same tensors and writes none
    assert lent.parts[1].tensor.data_ptr() == v.parts[1].tensor.data_ptr() and not lent.parts[1].writes and not lent.parts[0].parts[0].writes
    assert [tuple(t.shape) for t in st.state_tensors()] == [(2, 6), (2, 2, 3), (2, 4)]
    assert st.total_bytes() == 4 * (pool.numel() + 12 + 12 + 8)


# ----------------------------------------------------------------------------------- the plain mechanisms by hand

def test_delta_rule_by_hand_and_carried_state():
    # one head, a state of one row and one column, k = 1: F = g S, then S = F + beta (v - F), read by q
    one = lambda *a: np.array(a, dtype=float).reshape(-1, 1, 1)
    g, beta, v, q = one(0.5, 0.5, 1.0), np.array([[1.0], [0.5], [0.25]]), one(2.0, 4.0, -1.0), one(1.0, 3.0, 1.0)
    o, S = P.delta_scan(q, one(1, 1, 1), v, g, beta)
    s0 = 2.0
    s1 = 0.5 * s0 + 0.5 * (4.0 - 0.5 * s0)
    s2 = s1 + 0.25 * (-1.0 - s1)
    assert np.allclose(o.ravel(), [s0, 3 * s1, s2]) and np.allclose(S.ravel(), [s2])
    o2, S2 = P.delta_scan(q[1:], one(1, 1), v[1:], g[1:], beta[1:], state=np.array([[[s0]]]))
    assert np.allclose(o2, o[1:]) and np.allclose(S2, S)


def test_a_second_write_to_the_same_key_replaces_the_first():
    k = np.zeros((3, 1, 4))
    k[:, 0, 1] = 1.0
    v = np.arange(6.0).reshape(3, 1, 2)
    ones = np.ones((3, 1))
    o, S = P.delta_scan(k, k, v, ones[:, :, None], ones)
    assert np.allclose(o, v) and np.allclose(S[0, 1], v[2, 0]) and np.allclose(np.delete(S[0], 1, 0), 0.0)
    o, S = P.gated_scan(k, k, v, np.ones((3, 1, 4)))                            # the gated recurrence adds up
    assert np.allclose(S[0, 1], v.sum(0)[0])


def test_decays_act_on_the_rows_of_their_key_channel():
    k = np.array([[[1.0, 1.0]], [[0.0, 0.0]]])
    v = np.array([[[3.0]], [[0.0]]])
    g = np.array([[[1.0, 1.0]], [[0.5, 0.25]]])
    for S in (P.gated_scan(k, k, v, g)[1], P.delta_scan(k, k, v, g, np.ones((2, 1)))[1]):
        assert np.allclose(S[0, :, 0], [1.5, 0.75])


def test_convolution_unit_vectors_rotation_and_window_by_hand():
    u = np.array([[1.0], [2.0], [3.0], [4.0]])
    taps = np.array([[10.0, 100.0, 1.0]])
    y = P.causal_conv(u, taps)
    assert np.allclose(y[:, 0], [1.0, 102.0, 213.0, 324.0]) and np.allclose(P.causal_conv(u[2:], taps, before=u[:2]), y[2:])
    assert np.allclose(P.unit_vector(np.array([3.0, 4.0]), 0.0), [0.6, 0.8])
    assert np.allclose(P.unit_vector(np.array([3e-4, 4e-4])), np.array([3e-4, 4e-4]) / math.sqrt(25e-8 + 1e-6))
    x = np.zeros((2, 1, 6))
    x[:, 0] = [1.0, 2.0, 3.0, 4.0, 5.0, 6.0]
    y = P.rotate_half(x, 4, 100.0, 4.0)
    assert np.allclose(y[0], x[0]) and np.array_equal(y[1, 0, 4:], x[1, 0, 4:])
    for i, f in enumerate([0.25, 0.25 * 100.0 ** -0.5]):
        a, b = x[1, 0, i], x[1, 0, i + 2]
        assert np.isclose(y[1, 0, i], a * math.cos(f) - b * math.sin(f)) and np.isclose(y[1, 0, i + 2], b * math.cos(f) + a * math.sin(f))
    v = np.arange(1.0, 7.0).reshape(6, 1, 1)
    z = np.zeros((6, 1, 1))
    assert np.allclose(P.windowed_attention(z, z, v, 1.0, 3).ravel(), [1.0, 1.5, 2.0, 3.0, 4.0, 5.0])
    assert np.allclose(P.windowed_attention(z, z, v, 1.0, None).ravel(), [1.0, 1.5, 2.0, 2.5, 3.0, 3.5])


def test_streams_by_hand():
    xs = np.array([[[1.0], [10.0]]])
    assert np.allclose(P.streams_read(xs, np.array([2.0, 0.5])), [[7.0]])
    mix = np.array([[1.0, 2.0], [3.0, 4.0]])                     # from, to
    got = P.streams_write(xs, np.array([[100.0]]), mix, np.array([0.5, -1.0]))
    assert np.allclose(got[0, :, 0], [1.0 + 30.0 + 50.0, 2.0 + 40.0 - 100.0])


def test_linear_frequency_scaling():
    from kappai_b200.config.schema import ConfigError, PartSpec
    from kappai_b200.parts.base import BuildEnv, make_part
    env = BuildEnv(torch.device("cpu"), torch.float32, 8)
    enc = make_part("position", PartSpec("rope", {"rotary_dim": 4, "theta": 100.0, "scaling": {"factor": 4.0}}), env)
    assert np.allclose(enc.cos[3].numpy(), np.cos(3 * np.array([0.25, 0.025])))
    plain = make_part("position", PartSpec("rope", {"rotary_dim": 4, "theta": 100.0}), env)
    assert np.allclose(plain.cos[3].numpy(), np.cos(3 * np.array([1.0, 0.1])))
    with pytest.raises(ConfigError):
        make_part("position", PartSpec("rope", {"rotary_dim": 4, "theta": 100.0, "scaling": {"factor": -1.0}}), env)


def test_the_bench_configurations_are_valid_models():
    """``bench.py --design gosulorn`` times these layer sizes: every one of them reads as a model with all three mixers whose
    last layer runs the first one's weights."""
    import importlib.util
    import os
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    spec = importlib.util.spec_from_file_location("bench_for_test", os.path.join(root, "bench.py"))
    bench = importlib.util.module_from_spec(spec)
    spec.loader.exec_module(bench)
    for name, width, H, G, hd, ff, *_ in bench.DESIGN_SIZES:
        m = _spec(bench.gosulorn_config(width, H, G, hd, ff))
        assert [l.mixer.kind for l in m.layers] == ["gated_delta", "gated_linear", "parallel"], name
        assert [e.layer for e in m.schedule] == [0, 1, 2, 0] and m.residual.params["streams"] == bench.GOSULORN_STREAMS
        left = m.layers[2].mixer.params["mixers"]["left"].params
        assert left["window"] == bench.GOSULORN_WINDOW and left["head_dim"] == left["value_dim"] == hd
