"""Gosulorn on the GPU: every new mechanism's kernel against the plain functions, the mixers and the layer arrangement as
parts in batches cut in two, then whole models through the step function, the trace runner and the engine in every way
of cutting the work."""
import copy
import math

import numpy as np
import pytest
import torch

import plain_gosulorn as P
import replay_util as R
from gosulorn_configs import CONFIGS, make_model_dir, make_weights, write_model_dir
from test_kernels_gpu import i32, rt
from tolerances import tol_for

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = [torch.float32, torch.bfloat16]


def dev(a, dtype=torch.float32):
    return torch.as_tensor(np.asarray(a), dtype=torch.float32).to(DEV).to(dtype).contiguous()


def host(t):
    return t.detach().double().cpu().numpy()


def close(got, want, dtype, tol16=0.02, tol32=3e-5):
    tol = tol32 if dtype == torch.float32 else tol16
    err = np.abs(got - want).max() / max(1.0, np.abs(want).max())
    assert err <= tol, err


def f32(a):
    return np.asarray(a, dtype=np.float32).astype(np.float64)


@pytest.fixture(scope="module")
def gos_dirs(tmp_path_factory):
    root = tmp_path_factory.mktemp("gosulorn")
    return {n: make_model_dir(n, str(root)) for n in CONFIGS}


@pytest.fixture(scope="module")
def gos_plain(gos_dirs):
    return {n: P.PlainGosulorn(d) for n, d in gos_dirs.items()}


def _chunk_lists(cu, rows):
    """(chunk_seg, chunk_row0, seg_chunk0, n_chunks) of segments with the row bounds ``cu`` in chunks of ``rows``."""
    seg, row0, first = [], [], [0]
    for i in range(len(cu) - 1):
        for r in range(int(cu[i]), int(cu[i + 1]), rows):
            seg.append(i)
            row0.append(r)
        first.append(len(seg))
    return i32(seg), i32(row0), i32(first), len(seg)


def _tables(pieces, slots):
    """Device tables of a launch over ``pieces`` = [(request, first row, rows)]."""
    cu = np.concatenate([[0], np.cumsum([n for _, _, n in pieces])])
    row_seg = np.concatenate([[j] * n for j, (_, _, n) in enumerate(pieces)])
    return cu, i32(row_seg), (i32(cu), i32([p for _, p, _ in pieces]), i32([slots[i] for i, _, _ in pieces]))


# ------------------------------------------------------------------------------------- the recurrence kernels

SIZES = [  # kernel, heads, q/k heads, key channels, value columns, a decay a key channel, delta rule
    ("scan", 4, 2, 16, 16, False, True), ("scan", 3, 1, 24, 40, True, True), ("scan", 5, 5, 5, 3, True, True),
    ("scan", 2, 2, 128, 64, False, True), ("scan", 2, 1, 256, 36, True, True), ("scan", 3, 3, 64, 33, True, False),
    ("scan", 1, 1, 1, 1, True, False), ("scan", 2, 2, 130, 20, True, False),
    ("chunks", 4, 2, 16, 16, False, True), ("chunks", 3, 1, 24, 40, True, True), ("chunks", 5, 5, 5, 3, True, True),
    ("chunks", 2, 2, 128, 64, False, True), ("chunks", 4, 2, 128, 128, True, True), ("chunks", 2, 1, 100, 36, True, True),
    ("chunks", 3, 1, 30, 256, False, True), ("chunks", 2, 1, 128, 256, True, True), ("chunks", 2, 2, 64, 9, False, True),
    ("chunks", 3, 3, 64, 33, True, False), ("chunks", 1, 1, 1, 1, True, False), ("chunks", 1, 1, 1, 1, False, True),
    ("chunks", 2, 2, 120, 96, True, False), ("chunks", 2, 2, 64, 256, True, False), ("chunks", 2, 2, 128, 128, True, False)]


def _recurrence_case(kernel, H, G, D, Pv, chan, delta, dtype, lens, cut, extra, draw_lg, rng, tol):
    """Requests of ``lens`` rows, the second from ``cut`` rows of an earlier launch, then one-row steps with the segments in
    another order than the slots; the slots held another request's state, which position 0 alone must wipe."""
    from kappai_b200.ops import kernels as K
    in_dt = torch.float32 if delta else dtype
    q_scale = 1.0 if delta else D ** -0.5
    slots = [2, 0, 3]
    state = torch.full((4, H * D * Pv + 5), 7.0, device=DEV)
    x = {}
    for i, L in enumerate(lens):
        n = L + extra
        unit = (lambda a: P.unit_vector(a)) if delta else (lambda a: a)
        x[i] = dict(q=rt(unit(rng.normal(0, 1, (n, G, D))), in_dt), k=rt(unit(rng.normal(0, 1, (n, G, D))), in_dt),
                    v=rt(rng.normal(0, 1, (n, H, Pv)), in_dt), lg=f32(draw_lg((n, H, D if chan else 1))), beta=f32(rng.uniform(0, 1, (n, H))))
    got = {i: np.zeros((lens[i] + extra, H, Pv)) for i in x}

    def launch(pieces):
        cu, _, seg = _tables(pieces, slots)
        part = lambda name: np.concatenate([x[i][name][p:p + n] for i, p, n in pieces])
        n = int(cu[-1])
        rows = dev(np.concatenate([part(name).reshape(n, -1) for name in ("q", "k", "v")], 1), in_dt)
        q, k, v = rows[:, :G * D], rows[:, G * D:2 * G * D], rows[:, 2 * G * D:]
        lg = dev(part("lg").reshape(n, -1))
        beta = dev(part("beta")) if delta else None
        out = torch.full((n, H * Pv), float("nan"), device=DEV)
        args = (len(pieces), H, G, D, Pv, chan, True)
        if kernel == "scan":
            K.recur_scan(q, k, v, lg, beta, q_scale, state, *seg, out, *args)
        else:
            K.recur_chunks(q, k, v, lg, beta, q_scale, state, *seg, *_chunk_lists(cu, K.recur_chunk_rows()), out, *args)
        o = host(out).reshape(n, H, Pv)
        for (i, p, m), r0 in zip(pieces, cu[:-1]):
            got[i][p:p + m] = o[r0:r0 + m]

    launch([(1, 0, cut)])
    launch([(0, 0, lens[0]), (1, cut, lens[1] - cut), (2, 0, lens[2])])
    for s in range(extra):
        launch([(2, lens[2] + s, 1), (0, lens[0] + s, 1), (1, lens[1] + s, 1)])
    for i in x:
        rep = lambda a: np.repeat(a, H // G, axis=1)
        g = np.exp(x[i]["lg"])
        q, k = rep(x[i]["q"]) * q_scale, rep(x[i]["k"])
        if delta:
            want, S = P.delta_scan(q, k, x[i]["v"], g, x[i]["beta"])
        else:
            want, S = P.gated_scan(q, k, x[i]["v"], np.broadcast_to(g, (len(g), H, D)))
        err = np.abs(got[i] - want).max() / max(1.0, np.abs(want).max())
        assert err <= tol, (i, err)
        s_err = np.abs(host(state)[slots[i], :H * D * Pv].reshape(H, D, Pv) - S).max() / max(1.0, np.abs(S).max())
        assert s_err <= tol, (i, s_err)
    assert torch.all(state[:, H * D * Pv:] == 7.0).item() and torch.all(state[1] == 7.0).item()      # what is not theirs stays


@pytest.mark.parametrize("kernel,H,G,D,Pv,chan,delta", SIZES)
def test_recurrence_kernels_segments_states_and_slots(kernel, H, G, D, Pv, chan, delta):
    rng = np.random.default_rng(H * 100 + D + Pv)
    for dtype in ([torch.float32] if delta else DTYPES):
        _recurrence_case(kernel, H, G, D, Pv, chan, delta, dtype, [65, 150, 1], 18, 4,
                         lambda s: -np.exp(rng.uniform(-6, 0.5, s)), rng, 2e-5)


@pytest.mark.parametrize("kernel", ["scan", "chunks"])
@pytest.mark.parametrize("chan,delta", [(False, True), (True, True), (True, False)])
def test_recurrence_with_decays_of_every_size(kernel, chan, delta):
    """Channels that keep everything beside channels that forget at once (a factor of exp(-60) a row: a chunk's sums of
    logarithms go far below what a float32 exponential holds): nothing overflows, and what is kept is right."""
    rng = np.random.default_rng(4)
    draw = lambda s: -np.exp(rng.uniform(-14, 4.1, s)) * rng.integers(0, 2, s)
    _recurrence_case(kernel, 2, 1, 48, 24, chan, delta, torch.float32, [130, 90, 40], 30, 2, draw, rng, 2e-5)


@pytest.mark.parametrize("kernel", ["scan", "chunks"])
@pytest.mark.parametrize("chan,delta", [(False, True), (True, True), (True, False)])
def test_a_far_write_counts(kernel, chan, delta):
    """A key of a direction of its own is written once, 2000 rows before its query, in another launch: what the query reads
    is that write's value times the decays between."""
    from kappai_b200.ops import kernels as K
    rng = np.random.default_rng(9)
    H, D, Pv, L, at = 2, 32, 16, 2100, 40
    k = rng.normal(0, 1, (L, H, D))
    k[:, :, 0] = 0.0
    k = P.unit_vector(k)
    k[at] = 0.0
    k[at, :, 0] = 1.0
    q = k.copy()
    q[-1] = 0.0
    q[-1, :, 0] = 1.0
    v, lg, beta = rng.normal(0, 1, (L, H, Pv)), np.full((L, H, D if chan else 1), -1e-4), np.ones((L, H))
    rows = dev(np.concatenate([a.reshape(L, -1) for a in (q, k, v)], 1))
    lgd, bd = dev(lg.reshape(L, -1)), dev(beta)
    state = torch.full((1, H * D * Pv), 3.0, device=DEV)
    out = torch.zeros((L, H * Pv), device=DEV)
    for a, b in ((0, 700), (700, 701), (701, L)):
        r = rows[a:b]
        seg = (i32([0, b - a]), i32([a]), i32([0]))
        args = (r[:, :H * D], r[:, H * D:2 * H * D], r[:, 2 * H * D:], lgd[a:b].contiguous(), bd[a:b].contiguous() if delta else None, 1.0,
                state, *seg)
        if kernel == "scan":
            K.recur_scan(*args, out[a:b], 1, H, H, D, Pv, chan)
        else:
            K.recur_chunks(*args, *_chunk_lists([0, b - a], K.recur_chunk_rows()), out[a:b], 1, H, H, D, Pv, chan)
    want = math.exp(-1e-4 * (L - 1 - at)) * v[at]
    got = host(out)[-1].reshape(H, Pv)
    # (the last row's own write, of its own key, adds v (k . q) = 0)
    assert np.abs(got - want).max() <= 2e-4, np.abs(got - want).max()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,Pv,taps,chan", [
    (4, 2, 16, 16, 3, False), (3, 1, 24, 40, 4, True), (5, 5, 5, 3, 2, True), (4, 4, 64, 128, 4, True), (2, 1, 128, 64, 1, False),
    (2, 2, 256, 36, 3, True), (3, 3, 132, 20, 4, False), (6, 3, 4, 8, 2, True), (2, 1, 8, 12, 7, False), (1, 1, 1, 1, 5, True)])
def test_what_stands_in_front_of_the_delta_rule(H, G, D, Pv, taps, chan, dtype):
    """Convolutions, silu, unit vectors, step sizes and decays: a whole prompt, a continuation, short and one-row segments
    in one launch, then one-row steps; kept inputs of another request in the slots."""
    from kappai_b200.ops import kernels as K
    rng = np.random.default_rng(D + taps)
    C, n_dec = 2 * G * D + H * Pv, H * D if chan else H
    conv_col, b_col = 8, 8 + -(-C // 8) * 8
    a_col, ld = b_col + H, -(-(b_col + 2 * H) // 8) * 8
    lens, cut, extra = [21, 40, 1, 2], 18, 3
    rows = {i: rt(rng.normal(0, 1, (L + extra, ld)), dtype) for i, L in enumerate(lens)}
    zs = {i: f32(rng.normal(0, 2, (L + extra, n_dec))) for i, L in enumerate(lens)}
    w_taps, a_log, dt_bias = f32(rng.normal(0, 1 / math.sqrt(taps), (C, taps))), rng.uniform(-2, 1, H), f32(rng.uniform(-4, 0, n_dec))
    neg_a = f32(-np.exp(a_log))
    slots = [2, 0, 3, 1]
    kept = torch.full((5, 11 + (taps - 1) * C), 7.0, device=DEV)
    got = {i: [None] * (L + extra) for i, L in enumerate(lens)}

    def launch(pieces):
        cu, row_seg, seg = _tables(pieces, slots)
        n = int(cu[-1])
        p = dev(np.concatenate([rows[i][a:a + m] for i, a, m in pieces]), dtype)
        out, beta = torch.full((n, C), float("nan"), device=DEV), torch.full((n, H), float("nan"), device=DEV)
        lg = dev(np.concatenate([zs[i][a:a + m] for i, a, m in pieces])) if chan else torch.full((n, H), float("nan"), device=DEV)
        K.delta_prep(p, conv_col, b_col, a_col, dev(w_taps), dev(neg_a), dev(dt_bias), kept[:, 11:], row_seg, *seg, out, beta, lg,
                     len(pieces), H, G, D, Pv, D ** -0.5, chan, all(m == 1 for _, _, m in pieces))
        for (i, a, m), r0 in zip(pieces, cu[:-1]):
            for j in range(m):
                got[i][a + j] = np.concatenate([host(t[r0 + j]) for t in (out, beta, lg)])

    launch([(1, 0, cut)])
    launch([(0, 0, lens[0]), (1, cut, lens[1] - cut), (2, 0, 1), (3, 0, 2)])
    for s in range(extra):
        launch([(3, 2 + s, 1), (0, lens[0] + s, 1), (2, 1 + s, 1), (1, lens[1] + s, 1)])
    for i, x in rows.items():
        T = len(x)
        y = P.silu(P.causal_conv(x[:, conv_col:conv_col + C], w_taps))
        q = P.unit_vector(y[:, :G * D].reshape(T, G, D)) * D ** -0.5
        k = P.unit_vector(y[:, G * D:2 * G * D].reshape(T, G, D))
        beta = P.sigmoid(x[:, b_col:b_col + H])
        z = zs[i] if chan else x[:, a_col:a_col + H]
        lg = np.repeat(neg_a, n_dec // H)[None, :] * P.softplus(z + dt_bias)
        want = np.concatenate([q.reshape(T, -1), k.reshape(T, -1), y[:, 2 * G * D:], beta, lg], 1)
        err = np.abs(np.stack(got[i]) - want) / np.maximum(1.0, np.abs(want))
        assert err.max() <= 1e-5, (i, err.max())
    assert torch.all(kept[:, :11] == 7.0).item() and torch.all(kept[4] == 7.0).item()


def test_prep_rows_have_the_same_bits_in_every_form():
    """A row in a step of many rows (four rows a lane) and alone (one row a warp)."""
    from kappai_b200.ops import kernels as K
    rng = np.random.default_rng(1)
    for H, G, D, Pv, taps in ((4, 2, 64, 32, 4), (2, 1, 132, 36, 3), (3, 3, 24, 20, 2)):
        C = 2 * G * D + H * Pv
        ld = C + 2 * H + (-(C + 2 * H)) % 8
        x = dev(rng.normal(0, 1, (40, ld)))
        w, na, db = dev(rng.normal(0, 1, (C, taps))), dev(-np.ones(H)), dev(np.zeros(H))
        mk = lambda n: (torch.empty((n, C), device=DEV), torch.empty((n, H), device=DEV), torch.empty((n, H), device=DEV))
        kept = torch.zeros((1, (taps - 1) * C), device=DEV)
        whole = mk(40)
        K.delta_prep(x, 0, C, C + H, w, na, db, kept, i32([0] * 40), i32([0, 40]), i32([0]), i32([0]), *whole, 1, H, G, D, Pv, 0.5, False, False)
        kept.zero_()
        for r in range(40):
            one = mk(1)
            K.delta_prep(x[r:r + 1], 0, C, C + H, w, na, db, kept, i32([0]), i32([0, 1]), i32([r]), i32([0]), *one, 1, H, G, D, Pv, 0.5, False, True)
            for a, b in zip(one, whole):
                assert torch.equal(a[0], b[r]), (H, D, r)


def test_logarithms_of_sigmoid_decays():
    from kappai_b200.ops import kernels as K
    z = np.concatenate([np.linspace(-90, 90, 2001), [0.0, 1e-30, -1e-30]])
    got = host(K.log_decay_sigmoid(dev(z), 16.0))
    want = -np.logaddexp(0.0, -f32(z)) / 16.0
    assert np.abs(got - want).max() <= 2e-7 * np.abs(want).max() and np.all(np.abs(got - want) <= 3e-6 * np.abs(want) + 1e-38)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("C,taps,bias,act", [(24, 3, False, None), (40, 4, True, "silu"), (7, 5, False, "silu"), (64, 1, True, None),
                                             (36, 2, False, None)])
def test_channel_convolution(C, taps, bias, act, dtype):
    from kappai_b200.ops import kernels as K
    rng = np.random.default_rng(C)
    lens, cut, extra, slots, col = [19, 33, 1], 14, 2, [2, 0, 1], 8
    ld = col + C + (-(col + C)) % 8
    rows = {i: rt(rng.normal(0, 1, (L + extra, ld)), dtype) for i, L in enumerate(lens)}
    w, b = f32(rng.normal(0, 1, (C, taps))), f32(rng.normal(0, 1, C))
    kept = torch.full((4, max(1, (taps - 1) * C)), 7.0, device=DEV)
    got = {i: np.zeros((L + extra, C)) for i, L in enumerate(lens)}

    def launch(pieces):
        cu, row_seg, seg = _tables(pieces, slots)
        out = torch.empty((int(cu[-1]), C), dtype=dtype, device=DEV)
        K.channel_conv(dev(np.concatenate([rows[i][a:a + m] for i, a, m in pieces]), dtype), col, dev(w), kept, row_seg, *seg, out,
                       len(pieces), all(m == 1 for _, _, m in pieces), True, act, dev(b) if bias else None)
        for (i, a, m), r0 in zip(pieces, cu[:-1]):
            got[i][a:a + m] = host(out)[r0:r0 + m]

    launch([(1, 0, cut)])
    launch([(0, 0, lens[0]), (1, cut, lens[1] - cut), (2, 0, 1)])
    for s in range(extra):
        launch([(2, 1 + s, 1), (1, lens[1] + s, 1), (0, lens[0] + s, 1)])
    for i, x in rows.items():
        want = P.causal_conv(x[:, col:col + C], w) + (b if bias else 0.0)
        close(got[i], P.silu(want) if act else want, dtype, tol16=0.01)


# ------------------------------------------------------------------------------------- streams

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,S,d", [(5, 3, 36), (40, 4, 64), (3, 1, 37), (70, 2, 4100), (9, 5, 160), (2, 8, 8200), (3, 6, 512), (4, 7, 2052)])
def test_streams_in_one_pass(n, S, d, dtype):
    from kappai_b200.ops import kernels as K
    rng = np.random.default_rng(n + d)
    xs, y = f32(rng.normal(0, 2, (n, S, d)) + 1.0), f32(rng.normal(0, 1, (n, d)))
    mix, out_w, in_w, w = f32(np.eye(S) + rng.normal(0, 0.3, (S, S))), f32(rng.normal(1, 0.5, S)), f32(rng.normal(0.3, 0.4, S)), f32(rng.normal(1, 0.2, d))
    new = P.streams_write(xs, y, mix, out_w)
    for centred in (True, False):
        norm = P.layer_norm if centred else (lambda a, b, e: P.unit_rms(a, e) * b)
        xt, yt, h = dev(xs), dev(y), torch.empty((n, d), dtype=dtype, device=DEV)
        K.streams_rows(xt, yt, dev(mix), dev(out_w), dev(in_w), dev(w), 1e-3, centred, h)
        close(host(xt), new, torch.float32, tol32=2e-6)
        assert torch.count_nonzero(yt).item() == 0                               # cleared for whoever adds into it next
        close(host(h), norm(P.streams_read(new, in_w), w, 1e-3), dtype, tol16=0.01)
        xt, yt = dev(xs), dev(y)
        K.streams_rows(xt, yt, dev(mix), dev(out_w))                             # nothing is read next
        close(host(xt), new, torch.float32, tol32=2e-6)
        rows = [n - 1, 0]
        h2 = torch.empty((2, d), dtype=dtype, device=DEV)
        K.streams_rows(xt, norm_w=dev(w), eps=1e-5, centred=centred, h=h2, rows=i32(rows))      # the sum of the streams, picked rows
        close(host(h2), norm(new.sum(1)[rows], w, 1e-5), dtype, tol16=0.01)
        h3 = torch.empty((n, d), dtype=dtype, device=DEV)
        K.streams_rows(xt, in_w=dev(in_w), norm_w=dev(w), eps=1e-5, centred=centred, h=h3)
        close(host(h3), norm(P.streams_read(new, in_w), w, 1e-5), dtype, tol16=0.01)
    e = f32(rng.normal(0, 1, (n, d)))
    x = K.streams_enter(dev(e), torch.empty((n, S, d), device=DEV))
    assert np.array_equal(host(x), np.repeat(e[:, None], S, axis=1))


# ------------------------------------------------------------------------------------- the mixers as parts

def _bind(part, rng, dtype, free=12):
    """Random weights in the part's declared shapes, decays from a few tokens to hundreds; the stored values as float64."""
    ws, vals = {}, {}
    for name, spec in part.weight_specs().items():
        shape = tuple(free if n < 0 else n for n in spec.shape)
        last = name.split(".")[-1]
        if last == "A_log":
            a = rng.uniform(-2.5, 0.0, shape)
        elif last == "dt_bias":
            a = rng.uniform(-5.0, -1.0, shape)
        elif name.endswith("decay_up.bias"):
            a = rng.uniform(0.0, 5.0, shape)
        elif spec.role == "norm":
            a = 1 + 0.2 * rng.standard_normal(shape)
        elif spec.role == "bias":
            a = 0.3 * rng.standard_normal(shape)
        elif spec.role == "stream":
            a = (np.eye(shape[0]) if len(shape) == 2 else 1.0 / shape[0]) + 0.2 * rng.standard_normal(shape)
        else:
            a = rng.standard_normal(shape) / math.sqrt(shape[-1])
        t = torch.as_tensor(a.astype(np.float32)).to(dtype if spec.role in ("matrix", "embedding") else torch.float32)
        ws[name], vals[name] = t.cuda(), t.double().numpy()
    part.bind(ws)
    return vals


DELTA_NAMES = {"beta_proj.weight": "b", "A_log": "A_log", "dt_bias": "dt_bias", "norm.weight": "norm", "out_proj.weight": "o",
               "decay_proj.weight": "a", "gate_proj.weight": "g", "decay_down.weight": "a1", "decay_up.weight": "a2", "decay_up.bias": "a2.b",
               "gate_down.weight": "g1", "gate_up.weight": "g2", "out_proj.bias": "o.b"}
for _n in "qkv":
    DELTA_NAMES.update({f"{_n}_proj.weight": _n, f"{_n}_conv.weight": f"{_n}.conv", f"{_n}_proj.bias": f"{_n}.b"})


def _run_part(kind, params, plain_fn, dtype, d, page=16, lens=(150, 70, 33), cuts=(1, 64, 31), tol16=0.05, names=None):
    """Three requests, each in two steps (all in one batch), one of them a single token then the rest."""
    from kappai_b200.config import PartSpec
    from kappai_b200.parts import make_part
    from test_parts_gpu import env_for, run_mixer_two_steps
    rng = np.random.default_rng(len(kind) + d + page)
    part = make_part("mixer", PartSpec(kind, params), env_for(dtype, 1024))
    w = _bind(part, rng, dtype)
    w = {(names or (lambda n: DELTA_NAMES[n]))(k): v for k, v in w.items()}
    hs = [rt(rng.normal(0, 1, (L, d)), dtype) for L in lens]
    outs = run_mixer_two_steps(part, hs, list(lens), list(cuts), page, dtype)
    for h, got in zip(hs, outs):
        close(got, plain_fn(h, w), dtype, tol16=tol16)
    return part


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,Pv,taps,d,scale,low", [
    (4, 2, 16, 24, 4, 64, 1.0, False), (3, 1, 24, 8, 3, 48, -0.7, True), (5, 5, 9, 7, 2, 37, 1.3, True), (2, 2, 128, 64, 4, 128, 1.0, False),
    (2, 1, 64, 128, 1, 256, 0.5, True), (2, 1, 200, 16, 5, 64, 1.0, True)])
def test_gated_delta_part(H, G, D, Pv, taps, d, scale, low, dtype):
    m = {"heads": H, "kv_heads": G, "dim": D, "vdim": Pv, "conv": taps}
    params = {"hidden_size": d, "num_heads": H, "num_qk_heads": G, "head_dim": D, "value_dim": Pv, "conv_kernel": taps, "norm_eps": 1e-5,
              "decay": "channel" if low else "head", "gate": "sigmoid" if low else "silu", "gate_rank": "low" if low else "full",
              "out_scale": scale}
    _run_part("gated_delta", params, lambda h, w: scale * P.delta_mixer(h, w, m, 1e-5, low), dtype, d)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,D,Pv,tau,d", [(4, 16, 24, 16.0, 64), (3, 24, 8, 1.0, 48), (5, 9, 7, 4.0, 37), (2, 128, 64, 16.0, 128), (2, 256, 16, 2.5, 64)])
def test_gated_linear_part(H, D, Pv, tau, d, dtype):
    m = {"heads": H, "dim": D, "vdim": Pv, "tau": tau}
    params = {"hidden_size": d, "num_heads": H, "head_dim": D, "value_dim": Pv, "tau": tau, "norm_eps": 1e-5}
    _run_part("gated_linear", params, lambda h, w: P.gla_mixer(h, w, m, 1e-5), dtype, d)


def _left_case(H, G, D, Pv, taps, window, rot, scale):
    m = {"heads": H, "kv_heads": G, "dim": D, "vdim": Pv, "scale": scale}
    if window:
        m["mask"] = {"size": window}
    pos = None
    if rot:
        m["rot"] = {"dims": rot[0], "base": rot[1], "scaling": {"factor": rot[2]}}
        pos = {"kind": "rope", "params": {"rotary_dim": rot[0], "theta": rot[1], "scaling": {"factor": rot[2]}}}
    params = {"num_heads": H, "num_kv_heads": G, "head_dim": D, "value_dim": Pv, "scale": scale, "qk_norm_eps": None, "bias": True,
              "conv_kernel": taps, "window": window, "position": pos, "softmax_weights": "float32"}
    return m, params


LEFT = [(4, 2, 16, 24, 3, 20, (8, 1000.0, 4.0), 0.35), (3, 3, 24, 8, 2, None, None, 0.2), (5, 1, 7, 7, 5, 2, (6, 50.0, 1.0), 0.5),
        (8, 2, 64, 64, 4, 100, (32, 10000.0, 8.0), 0.125), (4, 4, 128, 128, 1, 40, (128, 500.0, 2.0), 0.1), (16, 1, 32, 48, 3, 30, (16, 100.0, 3.0), 0.2),
        (2, 1, 128, 160, 3, 50, (32, 5000.0, 8.0), 0.09)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,Pv,taps,window,rot,scale", LEFT)
def test_attention_part_with_convolutions_biases_and_a_rotation(H, G, D, Pv, taps, window, rot, scale, dtype):
    m, params = _left_case(H, G, D, Pv, taps, window, rot, scale)
    d = 64 if D != 7 else 36
    part = _run_part("attention", dict(params, hidden_size=d, out_scale=1.4), lambda h, w: 1.4 * P.conv_attention(h, w, m), dtype, d,
                     page=16 if D != 64 else 64)
    assert part.vdim == Pv and part.hd >= max(D, Pv)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case,right,ls,rs,d", [(0, (4, 2, 12, 20, 4), 1.3, 0.6, 64), (1, (3, 3, 20, 28, 2), 0.7, 1.0, 48), (3, (2, 1, 64, 32, 3), 1.0, -0.4, 128)])
def test_mixers_side_by_side(case, right, ls, rs, d, dtype):
    ml, pl = _left_case(*LEFT[case])
    H, G, D, Pv, taps = right
    m = {"left": ml, "left_scale": ls, "right": {"heads": H, "kv_heads": G, "dim": D, "vdim": Pv, "conv": taps}, "right_scale": rs}
    pr = {"hidden_size": d, "num_heads": H, "num_qk_heads": G, "head_dim": D, "value_dim": Pv, "conv_kernel": taps, "norm_eps": 1e-5,
          "decay": "channel", "gate": "sigmoid", "gate_rank": "low", "out_scale": rs}
    params = {"mixers": {"left": {"kind": "attention", "params": dict(pl, hidden_size=d, out_scale=ls)}, "right": {"kind": "gated_delta", "params": pr}}}
    name = lambda n: n.split(".", 1)[0] + "." + DELTA_NAMES[n.split(".", 1)[1]]
    part = _run_part("parallel", params, lambda h, w: P.parallel_mixer(h, w, m, 1e-5), dtype, d, names=name)
    assert part.graph_safe and len(part.joined) == 2 and part.mixers["left"].w_qkv is None        # one product for both


# ------------------------------------------------------------------------------------- whole models

_PLAIN = {}


def _requests(name, lengths, seed):
    rng = np.random.default_rng(seed)
    return {f"r{i}": rng.integers(0, CONFIGS[name][0]["vocab"], n).tolist() for i, n in enumerate(lengths)}


def _expect(plain, name, toks):
    key = (name, tuple(toks))
    if key not in _PLAIN:
        _PLAIN[key] = plain.forward(toks)
    return _PLAIN[key]


# lengths above the longest window of every model plus the decoded tail, a request of two or three tokens, lengths that end on
# and one behind a page's last token and a chunk's (64 rows)
LENGTHS = {"A": [150, 3, 64, 49], "B": [130, 41, 2, 97], "C": [77, 20, 101], "D": [330, 65, 129], "E": [140, 64, 90]}
PROMPTS = {"A": [30, 1, 60, 48], "B": [50, 40, 1, 80], "C": [40, 19, 60], "D": [150, 3, 128], "E": [100, 63, 30]}
N_LAST = {"A": 110, "B": 60, "C": 40, "D": 170, "E": 70}
BF16_REL_RMS = 0.04    # a row's 16-bit error (rms over the vocabulary / the row's spread): 95 % of the rows; 99 % twice that
BF16_BETWEEN_CUTS = 0.06


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name,page_size", [("A", 16), ("B", None), ("C", 32), ("D", None), ("E", 8)])
def test_every_cut_agrees_with_plain(name, page_size, dtype, gos_dirs, gos_plain, tmp_path):
    """Whole prompts, the last tokens decoded one by one (more of them than the longest window), portions down to two
    tokens, and up to four requests mixed in a pool so small that pages and slots go round."""
    plain = gos_plain[name]
    reqs = _requests(name, LENGTHS[name], 31)
    prompt_len = dict(zip(reqs, PROMPTS[name]))
    expected = {rid: _expect(plain, name, t) for rid, t in reqs.items()}
    page = page_size or 64
    rounded = sorted(-(-len(t) // page) * page for t in reqs.values())
    max_tokens = rounded[-1] + rounded[0] + 2 * page          # the longest request and the shortest fit together, not all
    tr = R.Trace()
    R.whole(tr, reqs)
    R.last_decoded(tr, reqs, n_last=N_LAST[name])
    R.portions(tr, reqs)
    b = len(tr.steps)
    R.mixed(tr, reqs, prompt_len, seed=5, max_live=4, page=page, max_tokens=max_tokens)
    assert max(len(s["entries"]) for s in tr.steps[b:]) >= 2
    out = R.run_trace(gos_dirs[name], dtype, tr, str(tmp_path / "out"), max_tokens, page_size)
    rel = []
    for st, rows in zip(tr.steps, tr.rows):
        for j, (rid, pos) in enumerate(rows):
            e = expected[rid][pos]
            rel.append((float(np.sqrt(np.mean((out[st["step"]][j] - e) ** 2)) / e.std()), st["step"], rid, pos))
    r = np.array([x[0] for x in rel])
    print(f"{name} {dtype}: {len(r)} rows, relative rms error median {np.median(r):.2e}, 95 % {np.quantile(r, 0.95):.2e}, worst {r.max():.2e}")
    if dtype == "bfloat16":
        assert np.quantile(r, 0.95) <= BF16_REL_RMS and np.quantile(r, 0.99) <= 2 * BF16_REL_RMS, max(rel)
        apart = []
        for place, rows in R.rows_by_place(tr, out).items():
            e = expected[place[0]][place[1]]
            apart.append(max(float(np.sqrt(np.mean((x - rows[0]) ** 2)) / e.std()) for x in rows[1:]))
        assert np.quantile(apart, 0.99) <= BF16_BETWEEN_CUTS, max(apart)
    else:
        assert r.max() <= 1e-4, max(rel)
    stats = R.cache_stats(str(tmp_path / "out"))
    assert stats and all(g["reused"] > 0 and g["handed_out"] > g["pages"] for g in stats.values()), stats
    if dtype == "float32":
        for place, rows in R.rows_by_place(tr, out).items():
            assert len(rows) >= 2, place
            for x in rows[1:]:
                assert np.array_equal(rows[0], x), f"{name}: float32 logits of {place} differ between cuts"


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_residual_after_every_layer_run(name, gos_dirs, gos_plain):
    """What an observer sees is the sum of the streams, behind every layer run (those with another layer's weights too)."""
    from kappai_b200 import ModelRunner, StepEntry
    plain = gos_plain[name]
    toks = _requests(name, [57], 8)["r0"]
    want = []
    plain.forward(toks, want)
    r = ModelRunner(gos_dirs[name], dtype="float32", max_tokens=256, max_requests=2, cuda_graphs=False)
    got = []
    r.observer = lambda i, x: got.append(x.detach().cpu().numpy().copy())
    r.step([StepEntry("a", toks, [0])])
    assert len(got) == len(want) + 1 == len(CONFIGS[name][0]["layers"]) + 1
    for i, w in enumerate(want):
        assert np.abs(got[i + 1] - w).max() < 1e-4 * max(1.0, np.abs(w).max()), (i, np.abs(got[i + 1] - w).max())


def test_a_window_one_token_off_or_a_lost_state_would_show(gos_plain, tmp_path):
    """Model A with scores so large that a softmax row sits on one or two keys and with slow decays: the plain model with every
    window one token longer or shorter, with a convolution that starts empty in the middle, or with states that do, is far
    away at many positions; the engine is not, for tokens of a prompt, of portions of it and for tokens decoded one by one."""
    from kappai_b200 import ModelRunner, StepEntry
    cfg = copy.deepcopy(CONFIGS["A"][0])
    for layer in cfg["layers"]:
        if layer["type"] == "parallel":
            layer["mixer"]["left"]["scale"] = 3.0
    weights = make_weights(cfg, 17)
    for n in weights:
        if n.endswith("dt_bias"):
            weights[n] = weights[n] - 3.0
    d = write_model_dir(cfg, weights, str(tmp_path / "peaked"))
    plain = P.PlainGosulorn(d)
    toks = np.random.default_rng(3).integers(0, cfg["vocab"], 140).tolist()
    want = plain.forward(toks)
    rel = lambda a, b: np.sqrt(((a - b) ** 2).mean(1)) / b.std(1)
    for delta in (1, -1):
        off = copy.deepcopy(cfg)
        for layer in off["layers"]:
            if layer["type"] == "parallel":
                layer["mixer"]["left"]["mask"]["size"] += delta
        assert (rel(P.PlainGosulorn(config=off, tensors=plain.w).forward(toks), want) > 0.1).sum() >= 20, delta
    late = plain.forward(toks[60:])                              # what a request that forgot its first 60 tokens would give
    assert (rel(late[40:], want[100:]) > 0.1).sum() >= 30        # (40 tokens on, beyond every window: the states alone)
    no_conv = {k: (np.where(np.arange(v.shape[1]) == v.shape[1] - 1, v, 0.0) if k.endswith(".conv") else v) for k, v in plain.w.items()}
    assert (rel(P.PlainGosulorn(config=cfg, tensors=no_conv).forward(toks), want) > 0.1).sum() >= 100
    r = ModelRunner(d, dtype="float32", max_tokens=256, max_requests=2, page_size=16, cuda_graphs=False)
    got = [r.step([StepEntry("a", toks[:37], list(range(37)))]).cpu().numpy()]
    got.append(r.step([StepEntry("a", toks[37:60], list(range(23)))]).cpu().numpy())
    for t in toks[60:]:
        got.append(r.step([StepEntry("a", [t], [0])]).cpu().numpy())
    err = rel(np.concatenate(got, 0), want)
    assert err.max() < 2e-4, (int(err.argmax()), err.max())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_batched_requests_equal_each_alone_and_captured_steps_equal_eager(dtype, gos_dirs):
    """Unequal requests decode together for many steps (the steps are captured into CUDA graphs on the way); every row
    equals the row of the request run alone without graphs."""
    from kappai_b200 import ModelRunner, StepEntry
    n_dec = 40
    reqs = _requests("A", [61 + n_dec, 9 + n_dec, 30 + n_dec], 12)

    def run(runner, group):
        out = {rid: [] for rid in group}
        lg = runner.step([StepEntry(rid, reqs[rid][:len(reqs[rid]) - n_dec], [len(reqs[rid]) - n_dec - 1]) for rid in group])
        for j, rid in enumerate(group):
            out[rid].append(lg[j].cpu().numpy().copy())
        for s in range(n_dec):
            lg = runner.step([StepEntry(rid, [reqs[rid][len(reqs[rid]) - n_dec + s]], [0]) for rid in group])
            for j, rid in enumerate(group):
                out[rid].append(lg[j].cpu().numpy().copy())
        for rid in group:
            runner.end(rid)
        return out

    r1 = ModelRunner(gos_dirs["A"], dtype=dtype, max_tokens=512, max_requests=4, page_size=16)
    together = run(r1, list(reqs))
    assert r1.model.graph_safe and r1.graphs is not None and len(r1.graphs.graphs) >= 1
    alone_runner = ModelRunner(gos_dirs["A"], dtype=dtype, max_tokens=512, max_requests=4, page_size=16, cuda_graphs=False)
    for rid in reqs:
        alone = run(alone_runner, [rid])[rid]
        for a, b in zip(alone, together[rid]):
            if dtype == "float32":
                assert np.array_equal(a, b)
            else:
                assert np.abs(a - b).max() <= 2 * tol_for(dtype, a)


@pytest.mark.parametrize("name", ["A", "B", "D"])
def test_a_slot_and_pages_used_again_start_empty(name, gos_dirs):
    """One slot and just enough pages for one request: a second request takes the slot and the pages of the first and gives
    what it gives alone."""
    from kappai_b200 import ModelRunner, StepEntry
    rng = np.random.default_rng(2)
    V = CONFIGS[name][0]["vocab"]
    a, b = rng.integers(0, V, 60).tolist(), rng.integers(0, V, 45).tolist()
    mk = lambda: ModelRunner(gos_dirs[name], dtype="float32", max_tokens=64, max_requests=1, page_size=16, cuda_graphs=False)
    r = mk()
    r.step([StepEntry("a", a, [len(a) - 1])])
    r.end("a")
    parts = [b[:1], b[1:8], b[8:]]
    second = [r.step([StepEntry("b", p, [len(p) - 1])]).cpu().numpy().copy() for p in parts]
    fresh = mk()
    for p, s in zip(parts, second):
        assert np.array_equal(s, fresh.step([StepEntry("x", p, [len(p) - 1])]).cpu().numpy())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(dtype, gos_dirs, gos_plain):
    """Six hundred tokens one by one behind a prompt of three: what a state gathers over them does not drift."""
    from kappai_b200 import ModelRunner, StepEntry
    toks = _requests("A", [603], 5)["r0"]
    want = _expect(gos_plain["A"], "A", toks)
    r = ModelRunner(gos_dirs["A"], dtype=dtype, max_tokens=640, max_requests=1, page_size=32)
    r.step([StepEntry("a", toks[:3], [])])
    rel = []
    for i in range(3, len(toks)):
        g = r.step([StepEntry("a", [toks[i]], [0])]).cpu().numpy()[0]
        rel.append(float(np.sqrt(((g - want[i]) ** 2).mean()) / want[i].std()))
    assert max(rel[-100:]) <= (1e-4 if dtype == "float32" else 2 * BF16_REL_RMS), (max(rel), max(rel[-100:]))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "D"])
def test_greedy_generation_through_the_engine(name, dtype, gos_dirs, gos_plain):
    from kappai_b200 import Engine, EngineArgs, SamplingParams
    plain = gos_plain[name]
    prompts = list(_requests(name, [5, 26, 60], 21).values())
    n_new = 40
    eng = Engine(EngineArgs(model=gos_dirs[name], dtype=dtype, max_batch=4, max_step_tokens=24, page_size=16, kv_tokens=1024))
    outs = eng.generate(prompts, SamplingParams(temperature=0.0, n_predict=n_new))
    assert [len(o) for o in outs] == [n_new] * len(prompts)
    for p, o in zip(prompts, outs):
        lg = plain.forward(p + o)[len(p) - 1:-1]
        for j, t in enumerate(o):
            best = int(np.argmax(lg[j]))
            assert t == best or lg[j][best] - lg[j][t] <= 4 * tol_for(dtype, lg[j]), (j, t, best)
    assert eng.runner.cache.slots.n_free == 4 and all(p.n_free == p.n_pages for p in eng.runner.cache.pools.values())


def test_command_line_and_random_weights(gos_dirs, gos_plain, tmp_path):
    """The command line runs the design like any other: greedy tokens equal the plain model's, --time names the design's
    kernels, and --random-weights writes a loadable model folder from a Gosulorn config.json."""
    import json
    import os
    import subprocess
    import sys
    plain = gos_plain["A"]
    prompt = _requests("A", [30], 77)["r0"]
    cmd = [sys.executable, "-m", "kappai_b200.cli", "-m", gos_dirs["A"], "-p", ",".join(map(str, prompt)), "-n", "12", "-t", "0",
           "--fp32", "--time"]
    p = subprocess.run(cmd, cwd=R.ROOT, capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    out = [int(t) for t in p.stdout.split()]
    assert len(out) == 12
    lg = plain.forward(prompt + out)[len(prompt) - 1:-1]
    for j, t in enumerate(out):
        best = int(np.argmax(lg[j]))
        assert t == best or lg[j][best] - lg[j][t] <= 1e-4 * max(1.0, np.abs(lg[j]).max()), (j, t, best)
    for name in ("streams_rows", "delta_prep", "recur_scan delta", "recur_scan gated", "channel_conv", "log_decay_sigmoid", "qk_norm_rope_kv"):
        assert name in p.stderr, (name, p.stderr[-3000:])
    cfgp = tmp_path / "c.json"
    cfgp.write_text(json.dumps(CONFIGS["B"][0]))
    made = tmp_path / "rw"
    cmd = [os.path.join(R.ROOT, "bin", "kappai-cli"), "--random-weights", str(cfgp), "-s", "5", "-m", str(made), "-t", "0", "-n", "5",
           "1 2 3"]
    p = subprocess.run(cmd, cwd=str(tmp_path), capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert len(p.stdout.split()) == 5 and os.path.isfile(made / "model.safetensors")
