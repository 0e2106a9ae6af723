"""Small Ladedra configurations that differ in every size, constant and option, and a writer of model folders whose
weights are large enough that every sublayer moves the residual (with weights of 0.02 a wrong key, a pooled block left
out or a lost state would hide below the tolerances)."""
import json
import math
import os
import tempfile

import numpy as np


def _rot(dims, base, scaling=None):
    r = {"dims": dims, "base": base}
    if scaling is not None:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return r


def _latent(heads, dim, rot_dim, vdim, rank, base=10000.0, scaling=None, scale=None, rot=True):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank,
         "scale": scale if scale is not None else 1.5 / math.sqrt(dim + rot_dim)}
    if rot:
        m["rot"] = _rot(rot_dim, base, scaling)
    return {"type": "latent_attention", "mixer": m}


def _left(heads, kv_heads, dim, vdim, size, pool, softcap=None, rot=None, scale=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else 2.0 / math.sqrt(dim)}
    if size is not None:
        m["mask"] = {"size": size}
        if pool is not None:
            m["mask"]["pool"] = pool
    if softcap is not None:
        m["softcap"] = softcap
    if rot is not None:
        m["rot"] = _rot(*rot)
    return m


def _right(heads, dim, vdim, rot=None):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "decay": [1.0 - 2.0 ** (-2 - 5 * h / max(1, heads - 1)) for h in range(heads)]}
    if rot is not None:
        m["rot"] = _rot(*rot)
    return m


def _parallel(left, right, left_scale, right_scale):
    return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": left_scale, "right_scale": right_scale}}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(experts, top, ff, groups=None, scale=None, shared=None):
    r = {"experts": experts, "top": top}
    if groups is not None:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    if scale is not None:
        r["scale"] = scale
    m = {"kind": "moe", "expert": {"ff": ff}, "router": r}
    if shared is not None:
        m["shared"] = {"ff": shared}
    return m


def _model(vocab, width, scale, layers, eps=1e-5, max_positions=None):
    c = {"architecture": "Ladedra", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "norm": {"eps": eps},
         "layers": [dict(mixer, mlp=mlp) for mixer, mlp in layers]}
    if max_positions is not None:
        c["max_positions"] = max_positions
    return c


# A: every mixer and feed-forward; values wider than keys on the left, narrower in the latent layers; six experts in three
# groups of which two are kept; a rotation of half a head; YaRN frequencies of which some pairs are kept, some blended,
# some divided; a layer without a feed-forward
LAD_A = _model(211, 64, 1.7, [
    (_latent(3, 24, 8, 16, 20, 100.0, (4.0, 64, 8.0, 1.0)), _dense(40)),
    (_parallel(_left(4, 2, 16, 24, 20, 5, 4.0, (8, 1000.0)), _right(2, 12, 20, (12, 50.0)), 1.3, 0.6), _moe(6, 2, 24, (3, 2), 1.5, 20)),
    (_latent(2, 16, 16, 24, 40, 5000.0), None),
    (_parallel(_left(2, 1, 32, 16, 9, 3, 20.0, (32, 200.0)), _right(3, 16, 8, (8, 300.0)), 0.8, 1.2), _dense(56)),
], max_positions=512)
# B: the parallel layer first; blocks longer than the window they stand behind, and blocks of one position; three heads
# everywhere; keys wider than values; no groups, no router scale, no shared unit; one expert of three
LAD_B = _model(97, 48, 0.5, [
    (_parallel(_left(3, 3, 24, 8, 4, 9, 6.0, (24, 500.0)), _right(3, 8, 24, (4, 80.0)), 0.7, 1.0), _moe(3, 1, 40)),
    (_latent(3, 8, 4, 8, 12, 50.0, (2.5, 100, 4.0, 0.5)), _moe(4, 2, 32, (4, 4), 0.7)),
    (_parallel(_left(3, 1, 8, 16, 33, 1, 3.0, (6, 100.0)), _right(3, 20, 12), 1.0, 0.5), _dense(24)),
], eps=1e-6, max_positions=400)
# C: sizes the fast kernels refuse (an odd width, odd head sizes, odd ranks, a vocabulary smaller than a warp, five query heads
# on one key head); no soft cap; a window without pooled blocks; a window of one with blocks of two; every expert chosen
LAD_C = _model(19, 37, 1.0, [
    (_latent(5, 7, 2, 9, 11, 30.0, scale=0.6), _moe(3, 3, 20, (1, 1), 2.0, 12)),
    (_parallel(_left(5, 1, 8, 12, 7, None, None, (4, 60.0), 0.5), _right(1, 7, 5, (6, 40.0)), 1.5, 0.9), _dense(28)),
    (_parallel(_left(1, 1, 7, 7, 1, 2, 2.0), _right(2, 5, 9), 0.9, 0.8), _moe(4, 1, 28, (2, 1), None, 8)),
], eps=1e-3)
# D: widths at which the decode products stream their weights and the prompt products run on tcgen05; head sizes 64 and 128
# (tensor-core attention kernels); a window of two pages with blocks that straddle pages; twenty latent heads (more than
# one head group), a latent of 128 and one of 208; prompts whose steps reach the grouped tcgen05 expert tiles
LAD_D = _model(400, 512, 1.0, [
    (_latent(4, 64, 64, 64, 128, 10000.0, (8.0, 128, 16.0, 1.0)), _dense(1024)),
    (_parallel(_left(8, 2, 64, 64, 128, 24, 30.0, (64, 10000.0)), _right(4, 64, 64, (64, 1000.0)), 1.0, 0.7), _moe(8, 2, 256, (4, 2), 2.0, 256)),
    (_latent(20, 32, 16, 48, 208, 2000.0), _moe(8, 2, 256, (2, 1), 1.0)),
    (_parallel(_left(4, 4, 128, 128, 40, 7, 15.0, (128, 5000.0)), _right(8, 32, 32, (16, 100.0)), 0.6, 0.9), None),
], max_positions=1024)
# E: sixteen query heads on one key head (more than the split-key kernel shares); a latent of 272 (the widest form of the
# tensor-core pass), 33 latent heads; keys of 96 and values of 160 columns; three experts of five
LAD_E = _model(300, 256, 2.0, [
    (_latent(33, 16, 16, 16, 272, 700.0, (3.0, 200, 10.0, 2.0)), _moe(5, 3, 64, None, 1.2, 64)),
    (_parallel(_left(16, 1, 32, 32, 30, 8, 10.0, (32, 400.0)), _right(2, 128, 64, (128, 900.0)), 1.1, 0.4), _moe(9, 2, 128, (3, 1), 0.9)),
    (_latent(2, 64, 32, 160, 48, 10000.0), _dense(96)),
], max_positions=640)
# F: what may be left out is left out: no mask (every earlier key is read, the sink stays), no soft cap, no rotation anywhere,
# no groups, no shared unit
LAD_F = _model(64, 32, 1.0, [
    (_parallel(_left(2, 1, 16, 16, None, None), _right(2, 8, 8), 1.0, 1.0), _moe(4, 2, 16)),
    (_latent(2, 16, 4, 8, 20, rot=False), None),
])

CONFIGS = {"A": (LAD_A, 3), "B": (LAD_B, 4), "C": (LAD_C, 5), "D": (LAD_D, 6), "E": (LAD_E, 7), "F": (LAD_F, 8)}


def tensor_shapes(cfg):
    d, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, d), "final.norm": (d,), "head": (V, d)}
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}."
        out.update({p + "norm1": (d,), p + "ls1": (d,), p + "rg1": (d, d), p + "rg1.b": (d,)})
        if layer["type"] == "latent_attention":
            H, dim, rd, vdim, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            out.update({p + "mix.q": (H * (dim + rd), d), p + "mix.dkv": (r + rd, d), p + "mix.dkv.norm": (r,), p + "mix.uk": (H * dim, r),
                        p + "mix.uv": (H * vdim, r), p + "mix.g": (H * vdim, d), p + "mix.o": (d, H * vdim)})
        else:
            l, r = m["left"], m["right"]
            H, G, dim, vdim = l["heads"], l["kv_heads"], l["dim"], l["vdim"]
            for n, sz in (("q", H * dim), ("k", G * dim), ("v", G * vdim)):
                out[p + f"mix.left.{n}"], out[p + f"mix.left.{n}.b"] = (sz, d), (sz,)
            out.update({p + "mix.left.sink": (H,), p + "mix.left.o": (d, H * vdim)})
            H, dim, vdim = r["heads"], r["dim"], r["vdim"]
            for n, sz in (("q", H * dim), ("k", H * dim), ("v", H * vdim), ("g", H * vdim)):
                out[p + f"mix.right.{n}"] = (sz, d)
            out[p + "mix.right.o"] = (d, H * vdim)
        mlp = layer["mlp"]
        if mlp is None:
            continue
        out.update({p + "norm2": (d,), p + "ls2": (d,), p + "rg2": (d, d), p + "rg2.b": (d,)})
        if mlp["kind"] == "dense":
            out.update({p + "mlp.up": (mlp["ff"], d), p + "mlp.down": (d, mlp["ff"])})
            continue
        out[p + "mlp.router"] = (mlp["router"]["experts"], d)
        units = [(f"e{e}", mlp["expert"]["ff"]) for e in range(mlp["router"]["experts"])]
        if mlp.get("shared"):
            units.append(("shared", mlp["shared"]["ff"]))
        for name, ff in units:
            out.update({p + f"mlp.{name}.gate": (ff, d), p + f"mlp.{name}.up": (ff, d), p + f"mlp.{name}.down": (d, ff)})
    return out


def make_weights(cfg, seed):
    """name -> bfloat16 tensor.  Matrices have unit gain (std 1/sqrt(inputs)), output matrices a gain of 2, the router
    a gain of 3, norm weights and layer scales 1 +- 0.2, biases 0 +- 0.5, sinks in [-1, 2], the embedding table std 1."""
    import torch
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        if name.endswith(".sink"):
            a = rng.uniform(-1.0, 2.0, shape)
        elif name.endswith(".b"):
            a = rng.normal(0.0, 0.5, shape)
        elif len(shape) == 1:
            a = 1.0 + rng.normal(0.0, 0.2, shape)
        elif name == "embed":
            a = rng.normal(0.0, 1.0, shape)
        else:
            gain = 2.0 if name.endswith((".o", ".down")) else (3.0 if name.endswith(".router") else 1.0)
            a = rng.normal(0.0, gain / math.sqrt(shape[1]), shape)
        out[name] = torch.from_numpy(a.astype(np.float32)).to(torch.bfloat16)
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
    return write_model_dir(cfg, make_weights(cfg, seed), tempfile.mkdtemp(prefix=f"lad_{name}_", dir=root))
