"""Ladedra without a GPU: the configuration reader and its errors, the tensor names and shapes of every test configuration,
what every layer keeps, page groups with an entry for several positions, and the plain mechanisms on cases worked out
by hand."""
import copy
import math

import numpy as np
import pytest
import torch

import plain_ladedra as P
from ladedra_configs import CONFIGS, make_weights, tensor_shapes, write_model_dir


def _spec(cfg):
    from kappai_b200.config.registry import config_from_dict
    arch, c = config_from_dict(cfg)
    assert arch.name == "Ladedra"
    return arch.build_spec(c)


def _model(cfg, dtype=torch.float32):
    from kappai_b200.engine.model import Model
    from kappai_b200.parts.base import BuildEnv
    return Model(_spec(cfg), BuildEnv(torch.device("cpu"), dtype, 32))


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_tensor_names_and_shapes(name):
    cfg = CONFIGS[name][0]
    table, want = _model(cfg).weight_table(), tensor_shapes(cfg)
    assert set(table) == set(want)
    for n, ws in table.items():
        assert ws.fits(want[n]), (n, ws.shape, want[n])
        assert not ws.fits(want[n] + (1,)) and not ws.fits(tuple(x + 1 for x in want[n]))


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_what_every_layer_keeps(name):
    from kappai_b200.cache import PagedKVSpec, StateSpec, leaf_specs
    cfg = CONFIGS[name][0]
    for layer, spec in zip(cfg["layers"], _model(cfg).cache_specs()):
        m, leaves = layer["mixer"], list(leaf_specs(spec))
        up = lambda n: -(-n // 16) * 16
        if layer["type"] == "latent_attention":
            # one row a token: the latent and the shared key part, nothing a head
            assert leaves == [PagedKVSpec(1, -(-(up(m["kv_rank"]) + up(m["rot_dim"])) // 64) * 64, planes=1)]
            continue
        left, right = m["left"], m["right"]
        mask = left.get("mask") or {}
        size, pool = mask.get("size"), mask.get("pool")
        assert leaves[0].num_kv_heads == left["kv_heads"] and leaves[0].head_dim >= max(left["dim"], left["vdim"]) and leaves[0].every == 1
        assert leaves[0].window == (size if pool is None else max(size, pool))
        assert leaves[-1] == StateSpec((right["heads"], right["dim"], right["vdim"]), "float32")
        assert len(leaves) == (2 if pool is None else 3)
        if pool is not None and pool > 1:
            assert leaves[1].every == pool and leaves[1].window is None and leaves[1].group_key != leaves[0].group_key


def test_parts_and_their_constants_come_from_the_configuration():
    cfg = CONFIGS["A"][0]
    m = _model(cfg)
    lat, par = m.blocks[0].mixer, m.blocks[1].mixer
    assert (lat.H, lat.dim, lat.rdim, lat.vdim, lat.rank) == (3, 24, 8, 16, 20) and lat.gated and lat.eps == cfg["norm"]["eps"]
    assert lat.scale == cfg["layers"][0]["mixer"]["scale"] and lat.rotary[2] == 8 and lat.rotary[3] is True
    assert lat.position.scaling == ("yarn", 4.0, 64.0, 8.0, 1.0, 100.0) and m.blocks[2].mixer.position.scaling is None
    left, right = par.mixers["left"], par.mixers["right"]
    assert (left.window, left.pool, left.cap, left.out_scale) == (20, 5, 4.0, 1.3) and left.norm_after and left.bias and not left.out_bias
    assert left.sink == "learned" and left.exact_weights and left.position.rotary_dim == 8 and not left.position.interleaved
    assert right.out_scale == 0.6 and right.k_scale == 12 ** -0.5 and right.activation is None and right.norm == "per_head" and right.gate == "silu"
    assert right.decay == cfg["layers"][1]["mixer"]["right"]["decay"]
    moe = m.blocks[1].ffn
    assert moe.groups == (3, 2) and moe.renormalise and moe.router_scale == 1.5 and moe.shared_ff == 20 and moe.routing == "softmax_all"
    assert not moe.correction and moe.activation == "silu"
    assert m.blocks[0].ffn.activation == "relu_squared" and m.blocks[2].ffn is None and m.blocks[2].sublayers == 1
    assert m.embedding.scale == 1.7 and not m.head.tied and m.graph_safe
    f = _model(CONFIGS["F"][0])
    bare = f.blocks[0].mixer.mixers["left"]
    assert bare.window is None and bare.pool is None and bare.cap == 0.0 and f.blocks[0].ffn.groups is None and f.blocks[0].ffn.router_scale == 1.0


@pytest.mark.parametrize("change,word", [
    (lambda c: c.pop("vocab"), "vocab"),
    (lambda c: c.pop("embedding"), "embedding"),
    (lambda c: c["embedding"].pop("scale"), "embedding.scale"),
    (lambda c: c["norm"].pop("eps"), "norm.eps"),
    (lambda c: c["layers"][0].update(type="attention"), "type"),
    (lambda c: c["layers"][0]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=10), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].update(factor=0), "factor"),
    (lambda c: c["layers"][0]["mlp"].pop("ff"), "mlp.ff"),
    (lambda c: c["layers"][0]["mlp"].update(kind="glu"), "kind"),
    (lambda c: c["layers"][1]["mixer"].pop("left_scale"), "left_scale"),
    (lambda c: c["layers"][1]["mixer"].pop("right"), "right"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=3), "kv_heads"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(softcap=-1.0), "softcap"),
    (lambda c: c["layers"][1]["mixer"]["left"]["mask"].update(pool=0), "mask.pool"),
    (lambda c: c["layers"][1]["mixer"]["left"]["mask"].update(size=0), "mask.size"),
    (lambda c: c["layers"][1]["mixer"]["right"]["decay"].pop(), "decay"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=7), "top"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=4), "count"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(keep=4), "keep"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=5), "top"),
])
def test_configuration_errors_name_the_key(change, word):
    from kappai_b200.config.schema import ConfigError
    cfg = copy.deepcopy(CONFIGS["A"][0])
    change(cfg)
    with pytest.raises(ConfigError) as e:
        _spec(cfg)
    assert word in str(e.value)


def test_loading_checks_shapes_and_the_padded_matrices(tmp_path):
    from kappai_b200.weights.loader import WeightError, load_weights
    cfg, seed = CONFIGS["A"]
    w = make_weights(cfg, seed)
    m = _model(cfg)
    load_weights(m, write_model_dir(cfg, w, str(tmp_path / "a")))
    lat = m.blocks[0].mixer
    uk = w["l0.mix.uk"].float().reshape(3, 24, 20)
    assert lat.w_uk_t.shape == (3, 32, 32) and torch.equal(lat.w_uk_t[:, :20, :24], uk.transpose(1, 2))
    assert not lat.w_uk_t[:, 20:].any() and not lat.w_uk_t[:, :, 24:].any()
    # the mixer's first product and the gate's rows are one matrix, and the block owns it
    blk = m.blocks[0]
    assert lat.w_in is None and torch.equal(blk.w_in[blk.cols:blk.cols + 64], w["l0.rg1"].float()) and torch.equal(blk.b_in[blk.cols:blk.cols + 64], w["l0.rg1.b"].float())
    assert not blk.b_in[:blk.cols].any()
    par = m.blocks[1]
    assert par.mixer.w_in is None and torch.equal(par.w_in[par.cols:], w["l1.rg1"].float()) and par.b_in[:par.cols].any()
    with pytest.raises(WeightError) as e:
        load_weights(_model(cfg), write_model_dir(cfg, dict(w, **{"l0.mix.dkv": w["l0.mix.dkv"][:-1]}), str(tmp_path / "b")))
    assert "l0.mix.dkv" in str(e.value)
    # what belongs to a feed-forward that a layer does not have may be there unread
    extra = {"l2.norm2": torch.ones(64).bfloat16(), "l2.ls2": torch.ones(64).bfloat16(), "l2.rg2": torch.ones(64, 64).bfloat16(),
             "l2.rg2.b": torch.ones(64).bfloat16()}
    load_weights(_model(cfg), write_model_dir(cfg, dict(w, **extra), str(tmp_path / "c")))


# ------------------------------------------------------------------ page groups with an entry for several positions

def test_a_pool_with_an_entry_for_several_positions():
    from kappai_b200.cache.manager import CacheManager, CacheError, PagePool
    pool = PagePool(6, 4, every=3)
    pool.open("a")
    assert [pool.pages_for(n) for n in (0, 2, 3, 12, 14, 15, 24, 26, 27)] == [0, 0, 1, 1, 1, 2, 2, 2, 3]
    pool.extend("a", 2)
    assert pool.table("a") == []
    pool.extend("a", 30)
    t = pool.table("a")
    assert len(t) == 3
    assert [pool.slot("a", p) for p in (0, 1, 2, 3, 5, 14, 29)] == [-1, -1, t[0] * 4, -1, t[0] * 4 + 1, t[1] * 4, t[2] * 4 + 1]
    pool.release_behind("a", 30)
    assert pool.n_free == 3
    pool.close("a")
    pool.check()
    with pytest.raises(CacheError):
        PagePool(4, 4, window=8, every=2)
    m = CacheManager({"t": (10, 4, 8), "p": (4, 4, None, None, 0, 5)}, 2)
    m.admit("x")
    m.extend("x", 37)
    got = m.token_slots("x", "p", 7, 30)
    assert got == [m.pools["p"].slot("x", p) for p in range(7, 37)] and sum(s >= 0 for s in got) == 6
    assert m.token_slots("x", "p", 37 - 2, 2) == [-1, -1]
    m.advance("x", 37)
    m.check()
    m.free("x")
    assert all(p.n_free == p.n_pages for p in m.pools.values())


def test_pool_sizes_hold_the_entries_of_any_mix_of_requests():
    """Requests whose page-rounded lengths together fill the pools always find pages for their entries."""
    from kappai_b200.engine.memory import GroupNeed, plan_cache
    rng = np.random.default_rng(0)
    for every, page in ((1, 16), (2, 16), (5, 8), (12, 64), (100, 16)):
        for _ in range(200):
            n = int(rng.integers(1, 5))
            lens = rng.integers(1, 300, n)
            tokens = sum(-(-int(L) // page) * page for L in lens)
            plan = plan_cache([GroupNeed("g", 4, every=every), GroupNeed("t", 4)], 0, 4, page, 4096, tokens, None)
            assert sum(-(-(int(L) // every) // page) for L in lens) <= plan.pages["g"], (every, page, lens)
            assert plan.pages["t"] * page == tokens
            if every > 4:
                assert plan.pages["g"] <= tokens // page // every + 4


def test_batches_accept_block_tables_of_entries():
    from kappai_b200.engine.batch import BatchError, Segment, lay_out_step
    seg = Segment("a", [1, 2, 3], 6, [2], 0, {"t": [0, 1, 2], "p": [5]}, {"t": [6, 7, 8], "p": [-1, -1, 20]})
    host = lay_out_step([seg], {"t": 4, "p": 4}, 10, 100, every={"t": 1, "p": 3})
    assert host.n_rows == 3
    with pytest.raises(BatchError):
        lay_out_step([seg], {"t": 4, "p": 4}, 10, 100)                # one entry a position would need three blocks
    with pytest.raises(BatchError):
        lay_out_step([Segment("a", [1, 2, 3], 12, [], 0, {"t": [0, 1, 2, 3], "p": [5]}, {"t": [1, 2, 3], "p": [-1, -1, 3]})],
                     {"t": 4, "p": 4}, 10, 100, every={"t": 1, "p": 3})


# ----------------------------------------------------------------------------------- the plain mechanisms by hand

def test_yarn_frequencies_by_hand():
    from kappai_b200.config.schema import ConfigError, PartSpec
    from kappai_b200.parts.base import BuildEnv, make_part
    sc = {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}
    f, m = P.yarn_frequencies(8, 100.0, sc)
    base = np.array([100.0 ** (-2 * i / 8) for i in range(4)])
    where = lambda t: 8 * math.log(64 / (2 * math.pi * t)) / (2 * math.log(100.0))
    lo, hi = max(math.floor(where(8.0)), 0), min(math.ceil(where(1.0)), 7)
    assert (lo, hi) == (0, 3)
    for i in range(4):
        r = min(max((i - lo) / (hi - lo), 0), 1)
        assert np.isclose(f[i], base[i] / 4 * r + base[i] * (1 - r))
    assert np.isclose(f[0], base[0]) and np.isclose(f[3], base[3] / 4) and np.isclose(m, 0.1 * math.log(4.0) + 1)
    env = BuildEnv(torch.device("cpu"), torch.float32, 40)
    enc = make_part("position", PartSpec("rope", {"rotary_dim": 8, "theta": 100.0, "pairing": "interleaved", "scaling": sc}), env)
    assert np.allclose(enc.cos[33].numpy(), m * np.cos(33 * f), atol=1e-6) and np.allclose(enc.sin[33].numpy(), m * np.sin(33 * f), atol=1e-6)
    # both edges at the same pair: the ramp is a step behind it
    f2, _ = P.yarn_frequencies(8, 100.0, dict(sc, fast=1.0001, slow=1.0, original=2 * math.pi * 100.0))
    enc2 = make_part("position", PartSpec("rope", {"rotary_dim": 8, "theta": 100.0, "scaling": dict(sc, fast=1.0001, slow=1.0, original=2 * math.pi * 100.0)}), env)
    assert np.allclose(enc2.sin[1].numpy(), m * np.sin(f2), atol=1e-6)
    with pytest.raises(ConfigError):
        make_part("position", PartSpec("rope", {"rotary_dim": 4, "theta": 100.0, "scaling": dict(sc, slow=0)}), env)


def test_rotation_by_hand():
    x = np.zeros((2, 1, 6))
    x[:, 0] = [1.0, 2.0, 3.0, 4.0, 5.0, 6.0]
    for inter, pairs in ((True, [(0, 1), (2, 3)]), (False, [(0, 2), (1, 3)])):
        y = P.rotate(x, {"dims": 4, "base": 100.0}, inter)
        assert np.allclose(y[0], x[0]) and np.array_equal(y[1, 0, 4:], x[1, 0, 4:])
        for i, (u, v) in enumerate(pairs):
            a = 100.0 ** (-2 * i / 4)
            assert np.isclose(y[1, 0, u], x[1, 0, u] * math.cos(a) - x[1, 0, v] * math.sin(a))
            assert np.isclose(y[1, 0, v], x[1, 0, v] * math.cos(a) + x[1, 0, u] * math.sin(a))


def test_pooled_window_by_hand():
    """A window of 4 and blocks of 3: row 7 sees tokens 4..7 and no token or block of 0..3 but block 0 (2 <= 7 - 4)."""
    tok, blk = P.pooled_window_masks(12, 4, 3)
    assert [int(x) for x in tok[7]] == [0, 0, 0, 0, 1, 1, 1, 1, 0, 0, 0, 0]
    assert [[int(b) for b in blk[i]] for i in (5, 6, 8, 9, 11)] == [[0] * 4, [1, 0, 0, 0], [1, 0, 0, 0], [1, 1, 0, 0], [1, 1, 0, 0]]
    v = np.arange(1.0, 13.0).reshape(12, 1, 1)
    z = np.zeros((12, 1, 1))
    o = P.pooled_attention(z, z, v, 1.0, 4, 3, None, None).ravel()
    assert np.isclose(o[5], (3 + 4 + 5 + 6) / 4) and np.isclose(o[6], (4 + 5 + 6 + 7 + 2) / 5)         # block 0's mean value is 2
    assert np.isclose(o[9], (7 + 8 + 9 + 10 + 2 + 5) / 6)
    o = P.pooled_attention(z, z, v, 1.0, 4, 3, None, np.array([math.log(3.0)])).ravel()
    assert np.isclose(o[9], (7 + 8 + 9 + 10 + 2 + 5) / 9)                                                # the sink counts as three keys
    assert np.allclose(P.softcap(np.array([0.0, 100.0, -100.0]), 2.0), [0.0, 2.0, -2.0])


def test_router_groups_by_hand():
    h = np.eye(6)[:1]
    z = np.log(np.array([[0.30, 0.02], [0.05, 0.20], [0.25, 0.18]]).reshape(-1))         # three groups of two experts
    router = np.zeros((6, 6))
    router[:, 0] = z
    idx, wt = P.route(h, router, {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 1}, "scale": 2.0})
    assert idx[0].tolist() == [0, 1] and np.allclose(wt[0], [2 * 0.30 / 0.32, 2 * 0.02 / 0.32])
    idx, wt = P.route(h, router, {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 2}})
    assert idx[0].tolist() == [0, 4] and np.allclose(wt[0], [0.30 / 0.55, 0.25 / 0.55])
    idx, _ = P.route(h, router, {"experts": 6, "top": 4, "groups": {"count": 3, "keep": 2}})
    assert idx[0].tolist() == [0, 4, 5, 1]
    idx, _ = P.route(h, router, {"experts": 6, "top": 4})
    assert idx[0].tolist() == [0, 4, 3, 5]
    assert np.isclose(P.choice_margin(h, router, {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 1}})[0], math.log(0.30 / 0.25))


def test_retention_and_the_gated_step_by_hand():
    d = 2
    w = {"q": np.eye(2)[:1], "k": np.eye(2)[:1], "v": np.eye(2)[1:], "g": np.array([[0.0, 0.0]]), "o": np.ones((d, 1))}
    h = np.array([[1.0, 2.0], [1.0, 4.0]])
    m = {"heads": 1, "dim": 1, "vdim": 1, "decay": [0.5]}
    assert np.allclose(P.retention(h, dict(w, g=np.array([[1.0, 0.0]])), m, 0.0), P.silu(np.ones((2, d))))   # o over its own size is 1
    x, y = np.array([[1.0, 1.0]]), np.array([[2.0, 4.0]])
    got = P.gated_step(x, np.array([[0.0, 0.0]]), y, np.array([3.0, 0.5]), np.eye(2), np.array([0.0, 50.0]))
    assert np.allclose(got, [[1 + 3 * 0.5 * 2, 1 + 0.5 * 4]])
    assert np.allclose(P.squared_relu_unit(np.array([[1.0, -2.0]]), {"up": np.eye(2), "down": np.eye(2)}), [[1.0, 0.0]])


def test_latent_attention_expanded_and_absorbed_are_the_same():
    """The plain mixer expands keys and values; the absorbed form (queries and sums against the latents) is equal."""
    rng = np.random.default_rng(0)
    m = {"heads": 2, "dim": 3, "rot_dim": 2, "vdim": 4, "kv_rank": 5, "scale": 0.7, "rot": {"dims": 2, "base": 10.0}}
    d, n = 6, 9
    w = {"q": (10, d), "dkv": (7, d), "uk": (6, 5), "uv": (8, 5), "g": (8, d), "o": (d, 8)}
    w = {k: rng.normal(0, 1, s) for k, s in w.items()}
    w["dkv.norm"] = rng.normal(1, 0.2, 5)
    h = rng.normal(0, 1, (n, d))
    q = (h @ w["q"].T).reshape(n, 2, 5)
    down = h @ w["dkv"].T
    c = P.rms(down[:, :5], 1e-5) * w["dkv.norm"]
    kr = P.rotate(down[:, None, 5:], m["rot"], True)[:, 0]
    qr = P.rotate(q[:, :, 3:], m["rot"], True)
    u = np.zeros((n, 2, 4))
    for x in range(2):
        qa = q[:, x, :3] @ w["uk"].reshape(2, 3, 5)[x]
        s = (qa @ c.T + qr[:, x] @ kr.T) * 0.7
        u[:, x] = (P.softmax_with_sink(s, np.tril(np.ones((n, n), bool))) @ c) @ w["uv"].reshape(2, 4, 5)[x].T
    want = (u.reshape(n, -1) * P.sigmoid(h @ w["g"].T)) @ w["o"].T
    assert np.allclose(P.latent_attention(h, w, m, 1e-5), want)


def test_step_tables_of_the_expanded_pass():
    from kappai_b200.engine.batch import StepSegments
    from kappai_b200.parts.latent import latent_tiles
    seg = lambda lens, pos: StepSegments(sum(lens), len(lens), np.concatenate([[0], np.cumsum(lens)]).astype(np.int32),
                                         np.array(pos, np.int32), list(lens), max(lens), all(n == 1 for n in lens))
    assert latent_tiles(seg([1, 4, 2], [7, 0, 9])) is None
    t = latent_tiles(seg([1, 2, 70, 3], [50, 9, 30, 5]))
    assert t.arrays["ctx_base"].tolist() == [0, 0, 0, 100, 108] and t.scalars["n_ctx"] == 108 and t.scalars["n_short_rows"] == 3
    assert t.arrays["tile_seg"].tolist() == [0, 1, 2, 2, 3] and t.arrays["tile_row0"].tolist() == [0, 1, 3, 67, 73]


def test_the_bench_configurations_are_valid_models():
    """``bench.py --design ladedra`` times these layer sizes: every one of them reads as a model with both mixers."""
    import importlib.util
    import os
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    spec = importlib.util.spec_from_file_location("bench_for_test", os.path.join(root, "bench.py"))
    bench = importlib.util.module_from_spec(spec)
    spec.loader.exec_module(bench)
    for name, width, H, G, hd, ff, E, top, ff_e, layers in bench.DESIGN_SIZES:
        m = _spec(bench.ladedra_config(width, H, G, hd, ff, E, top, ff_e, layers))
        assert {l.mixer.kind for l in m.layers} == {"latent_cache_attention", "parallel"}, name
        left = [l.mixer.params["mixers"]["left"].params for l in m.layers if l.mixer.kind == "parallel"][0]
        assert left["window"] == bench.LADEDRA_WINDOW and left["pool"] == bench.LADEDRA_POOL and left["softcap"] > 0
        assert m.layers[0].ffn.kind == "mlp" and m.layers[1].ffn.params["groups"]["count"] == 4
