"""Small Gosulorn configurations that differ in every size, constant and option, and a writer of model folders whose
weights are large enough that every sublayer moves the residual (with weights of 0.02 a wrong key, a lost state or a
window one token off would hide below the tolerances)."""
import copy
import json
import math
import os
import tempfile

import numpy as np


def _delta(heads, kv_heads, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def _left(heads, kv_heads, dim, vdim, conv, window=None, rot=None, scale=None):
    """rot: (dims, base) or (dims, base, factor)."""
    m = dict(_delta(heads, kv_heads, dim, vdim, conv), scale=scale if scale is not None else 1.0 / math.sqrt(dim))
    if window is not None:
        m["mask"] = {"size": window}
    if rot is not None:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
        if len(rot) > 2:
            m["rot"]["scaling"] = {"factor": rot[2]}
    return m


def _layer(kind, mixer, ff):
    return {"type": kind, "mixer": mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def _parallel(left, right, ls, rs, ff):
    return _layer("parallel", {"left": left, "left_scale": ls, "right": right, "right_scale": rs}, ff)


def _gla(heads, dim, vdim, tau, ff):
    return _layer("gla", {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}, ff)


def _again(layers, j):
    return dict(copy.deepcopy(layers[j]), weights_of=j)


def _model(vocab, width, streams, layers, eps=1e-5, max_positions=None):
    c = {"architecture": "Gosulorn", "vocab": vocab, "width": width, "streams": streams, "norm": {"eps": eps}, "layers": layers}
    if max_positions is not None:
        c["max_positions"] = max_positions
    return c


# A: every mixer, three layers run again with states of their own; values wider than keys on the left, both halves with
# shared keys; a window of 20
_L = [_parallel(_left(4, 2, 16, 24, 3, 20, (8, 1000.0, 4.0), 0.35), _delta(4, 2, 12, 20, 4), 1.3, 0.6, 40),
      _layer("delta", _delta(6, 3, 16, 8, 3), 72), _gla(2, 24, 16, 4.0, 48)]
GOS_A = _model(211, 64, 3, _L + [_again(_L, 1), _again(_L, 0), _again(_L, 2)])
# B: two streams; a layer without a feed-forward, run again; no window, no rotation; convolutions of one tap (nothing is kept
# of them) and of two; keys wider than values; every head with keys of its own; a chain of weights_of
_L = [_gla(3, 8, 24, 1.0, None), _parallel(_left(3, 3, 24, 8, 1), _delta(3, 3, 20, 28, 2), 0.7, 1.0, 56),
      _layer("delta", _delta(2, 2, 24, 24, 1), 16)]
_L = _L + [_again(_L, 0)]
GOS_B = _model(97, 48, 2, _L + [dict(copy.deepcopy(_L[0]), weights_of=3)], eps=1e-6, max_positions=400)
# C: sizes the fast kernels refuse (an odd width, odd heads, a vocabulary smaller than a warp, five query heads on one key
# head); one stream; a window of two; five taps; a rotation of all but one dimension without scaled frequencies; the
# right half's weight negative
GOS_C = _model(19, 37, 1, [_parallel(_left(5, 1, 7, 7, 5, 2, (6, 50.0)), _delta(5, 1, 9, 7, 6), 1.0, -0.8, 21),
                           _gla(1, 5, 3, 9.0, 12), _layer("delta", _delta(3, 1, 7, 5, 2), None)], eps=1e-3)
# D: widths at which the decode products stream their weights and the prompt products run on tcgen05; heads of 64 and 128
# (tensor-core attention, the wide form of the convolutions); four streams; a window of two pages
_L = [_layer("delta", _delta(4, 2, 128, 64, 4), 512),
      _parallel(_left(8, 2, 64, 64, 4, 128, (32, 10000.0, 8.0)), _delta(4, 4, 64, 128, 4), 0.9, 1.1, 256), _gla(4, 64, 128, 16.0, 512),
      _parallel(_left(4, 4, 128, 128, 2, 40, (128, 500.0, 2.0), 0.2), _delta(2, 1, 128, 128, 3), 1.0, 1.0, None)]
GOS_D = _model(400, 512, 4, _L + [_again(_L, 1)], max_positions=1024)
# E: the largest heads (256 channels of a key), sizes that are multiples of 4 but of nothing more, five streams, sixteen query
# heads on one key head
GOS_E = _model(300, 96, 5, [_layer("delta", _delta(2, 1, 256, 36, 3), 64), _gla(2, 160, 40, 2.5, 64),
                            _parallel(_left(16, 1, 32, 48, 2, 30, (16, 100.0, 3.0)), _delta(3, 3, 132, 20, 4), 1.1, 0.4, 100)],
               max_positions=640)

CONFIGS = {"A": (GOS_A, 3), "B": (GOS_B, 4), "C": (GOS_C, 5), "D": (GOS_D, 6), "E": (GOS_E, 7)}
RANKS = {"A": (5, 7), "B": (16, 3), "C": (3, 2), "D": (32, 64), "E": (24, 40)}      # of decays and of gates, in the tensors' shapes alone


def ranks_of(cfg):
    for name, (c, _) in CONFIGS.items():
        if c["width"] == cfg["width"]:
            return RANKS[name]
    return (8, 8)


def tensor_shapes(cfg):
    d, V, s = cfg["width"], cfg["vocab"], cfg["streams"]
    ra, rg = ranks_of(cfg)
    out = {"embed": (V, d), "final.norm": (d,)}

    def delta(p, m, low):
        H, G, D, Pv, K = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
        for n, rows in (("q", G * D), ("k", G * D), ("v", H * Pv)):
            out[p + n], out[p + n + ".conv"] = (rows, d), (rows, K)
        out.update({p + "b": (H, d), p + "A_log": (H,), p + "norm": (Pv,), p + "o": (d, H * Pv)})
        if low:
            out.update({p + "a1": (ra, d), p + "a2": (H * D, ra), p + "dt_bias": (H * D,), p + "g1": (rg, d), p + "g2": (H * Pv, rg)})
        else:
            out.update({p + "a": (H, d), p + "dt_bias": (H,), p + "g": (H * Pv, d)})

    for i, layer in enumerate(cfg["layers"]):
        if layer.get("weights_of") is not None:
            continue
        m, p = layer["mixer"], f"l{i}."
        subs = [1] if layer["mlp"] is None else [1, 2]
        for q in subs:
            out.update({f"{p}norm{q}": (d,), f"{p}hc{q}.in": (s,), f"{p}hc{q}.out": (s,), f"{p}hc{q}.mix": (s, s)})
        if layer["mlp"] is not None:
            ff = layer["mlp"]["ff"]
            out.update({p + "mlp.gate": (ff, d), p + "mlp.up": (ff, d), p + "mlp.down": (d, ff)})
        if layer["type"] == "delta":
            delta(p + "mix.", m, False)
        elif layer["type"] == "gla":
            H, D, Pv = m["heads"], m["dim"], m["vdim"]
            x = p + "mix."
            out.update({x + "q": (H * D, d), x + "k": (H * D, d), x + "v": (H * Pv, d), x + "g": (H * Pv, d), x + "o": (d, H * Pv),
                        x + "norm": (Pv,), x + "a1": (ra, d), x + "a2": (H * D, ra), x + "a2.b": (H * D,)})
        else:
            l, x = m["left"], p + "mix.left."
            for n, rows in (("q", l["heads"] * l["dim"]), ("k", l["kv_heads"] * l["dim"]), ("v", l["kv_heads"] * l["vdim"])):
                out[x + n], out[x + n + ".b"], out[x + n + ".conv"] = (rows, d), (rows,), (rows, l["conv"])
            out[x + "o"], out[x + "o.b"] = (d, l["heads"] * l["vdim"]), (d,)
            delta(p + "mix.right.", m["right"], True)
    return out


def make_weights(cfg, seed):
    """name -> bfloat16 tensor.  Matrices have unit gain (std 1/sqrt(inputs)), output matrices a gain of 2; norm weights 1 +-
    0.2; decays from a few tokens to hundreds; the stream coefficients read about the mean of the streams, write about
    one share to each and mix a sixth of every stream into the others; the embedding table std 1."""
    import torch
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        last = name.split(".")[-1]
        if ".hc" in name:
            s = shape[0]
            a = {"in": lambda: 1.0 / s + rng.normal(0, 0.3, shape), "out": lambda: 1.0 + rng.normal(0, 0.3, shape),
                 "mix": lambda: np.eye(s) + rng.normal(0, 0.15, shape)}[last]()
        elif last == "A_log":
            a = rng.uniform(-2.5, 0.0, shape)
        elif last == "dt_bias":
            a = rng.uniform(-5.0, -1.0, shape)
        elif name.endswith(".a2.b"):
            a = rng.uniform(0.0, 5.0, shape)
        elif last == "b" and len(shape) == 1:
            a = rng.normal(0, 0.4, shape)
        elif last == "conv":
            a = rng.normal(0, 1.0 / math.sqrt(shape[1]), shape)
        elif len(shape) == 1:
            a = 1.0 + rng.normal(0.0, 0.2, shape)
        elif name == "embed":
            a = rng.normal(0.0, 1.0, shape)
        else:
            a = rng.normal(0.0, (2.0 if last in ("o", "down") else 1.0) / math.sqrt(shape[1]), shape)
        out[name] = torch.from_numpy(np.asarray(a, dtype=np.float32)).to(torch.bfloat16)
    return out


def write_model_dir(cfg, weights, d):
    from kappai_b200.weights.safetensors_io import save_safetensors

    os.makedirs(d, exist_ok=True)
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_safetensors(os.path.join(d, "model.safetensors"), weights)
    return d


def make_model_dir(name, root=None):
    cfg, seed = CONFIGS[name]
    return write_model_dir(cfg, make_weights(cfg, seed), tempfile.mkdtemp(prefix=f"gos_{name}_", dir=root))
