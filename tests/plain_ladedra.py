"""A plain, slow Ladedra: whole sequences, no cache, one function for each mechanism.

Ladedra is a decoder-only model with pre-norm layers whose sublayers are scaled and gated,

    h = N(x) ;  x <- x + ls * sigmoid(W h + b) * f(h)

with N an RMS norm with a weight, ``ls`` a vector and (W, b) a matrix and a vector of the sublayer's own.  Two mixers:

* *latent_attention*: keys and values expanded from one normed low-rank latent a token, a rotated key part that all
  heads share (interleaved pairs, YaRN frequencies), causal softmax, a sigmoid gate on the concatenated heads;
* *parallel*: two mixers on the same input, summed with constant weights.  On the left grouped-query attention with
  biases whose rotated q and k are divided by their root mean square, with soft-capped scores and a learned sink in the
  softmax, over a sliding window and the means of all blocks of positions that lie wholly before it; on the right
  retention: a linear recurrence with a constant decay a head, rotated q and k.

The feed-forward is a square-of-relu unit or a mixture of silu units whose experts come from the best groups; the head
is a matrix of its own.

This file shares no code with the package: it reads config.json and the safetensors file itself, with numpy
only, and runs in float64.
"""
from __future__ import annotations

import json
import math
import os
import struct

import numpy as np


def read_safetensors(path):
    """name -> numpy array (bfloat16 widened exactly)."""
    with open(path, "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        header = json.loads(f.read(n))
        data = f.read()
    out = {}
    for name, e in header.items():
        if name == "__metadata__":
            continue
        b, en = e["data_offsets"]
        raw = data[b:en]
        if e["dtype"] == "BF16":
            a = (np.frombuffer(raw, dtype=np.uint16).astype(np.uint32) << 16).view(np.float32)
        elif e["dtype"] == "F32":
            a = np.frombuffer(raw, dtype=np.float32)
        else:
            raise ValueError(f"{name}: dtype {e['dtype']}")
        out[name] = a.reshape(e["shape"]).copy()
    return out


# ------------------------------------------------------------------- mechanisms

def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def yarn_frequencies(dims, base, scaling):
    """Rotary frequencies blended between interpolated (divided by the factor) and kept ones, pair by pair."""
    f = np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)])
    if not scaling:
        return f, 1.0
    factor, original = scaling["factor"], scaling["original"]

    def where(turns):                       # the (fractional) pair that turns this often over the original length
        return dims * math.log(original / (2 * math.pi * turns)) / (2 * math.log(base))

    lo = max(math.floor(where(scaling["fast"])), 0)
    hi = min(math.ceil(where(scaling["slow"])), dims - 1)
    ramp = np.clip((np.arange(dims // 2) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / factor * ramp + f * (1 - ramp), 0.1 * math.log(factor) + 1.0


def rotate(x, rot, interleaved, first_pos=0):
    """x [n, heads, width]: the first rot["dims"] entries of every head rotated by position; pairs (2i, 2i + 1) or
    (i, i + dims / 2)."""
    if not rot:
        return x
    dims = rot["dims"]
    f, m = yarn_frequencies(dims, rot["base"], rot.get("scaling"))
    a = (first_pos + np.arange(x.shape[0]))[:, None] * f[None, :]
    c, s = (np.cos(a) * m)[:, None, :], (np.sin(a) * m)[:, None, :]
    if interleaved:
        iu, iv = np.arange(0, dims, 2), np.arange(1, dims, 2)
    else:
        iu, iv = np.arange(dims // 2), np.arange(dims // 2) + dims // 2
    out = x.copy()
    u, v = x[..., iu], x[..., iv]
    out[..., iu] = u * c - v * s
    out[..., iv] = v * c + u * s
    return out


def softmax_with_sink(s, mask, sink=None):
    """Rows of ``exp(s_j) / (sum over visible j of exp(s_j) + exp(sink))``; ``sink`` None: a plain softmax."""
    s = np.where(mask, s, -np.inf)
    m = s.max(axis=-1, keepdims=True)
    if sink is not None:
        m = np.maximum(m, sink)
    e = np.where(mask, np.exp(s - m), 0.0)
    den = e.sum(axis=-1, keepdims=True)
    if sink is not None:
        den = den + np.exp(sink - m)
    return e / den


def softcap(s, cap):
    return s if not cap else cap * np.tanh(s / cap)


def latent_attention(h, w, m, eps):
    n = h.shape[0]
    H, dim, rd, vdim, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (h @ w["q"].T).reshape(n, H, dim + rd)
    down = h @ w["dkv"].T
    c = rms(down[:, :rank], eps) * w["dkv.norm"]
    kr = rotate(down[:, None, rank:], m.get("rot"), True)[:, 0]                  # one rotated part for all heads
    qr = rotate(q[:, :, dim:], m.get("rot"), True)
    k = (c @ w["uk"].T).reshape(n, H, dim)
    v = (c @ w["uv"].T).reshape(n, H, vdim)
    causal = np.arange(n)[:, None] >= np.arange(n)[None, :]
    out = np.zeros((n, H, vdim))
    for x in range(H):
        s = (q[:, x, :dim] @ k[:, x].T + qr[:, x] @ kr.T) * m["scale"]
        out[:, x] = softmax_with_sink(s, causal) @ v[:, x]
    return (out.reshape(n, -1) * sigmoid(h @ w["g"].T)) @ w["o"].T


def block_means(k, pool):
    """[n, G, d] -> the means of the whole blocks of ``pool`` rows, [n // pool, G, d]."""
    nb = k.shape[0] // pool
    return k[:nb * pool].reshape(nb, pool, *k.shape[1:]).mean(axis=1)


def pooled_window_masks(n, size, pool):
    """([n, n] tokens, [n, n // pool] blocks): row i sees token j if 0 <= i - j < size, and block b if its last
    position b pool + pool - 1 is at most i - size."""
    i = np.arange(n)[:, None]
    j = np.arange(n)[None, :]
    b = np.arange(n // pool)[None, :]
    return (j <= i) & (i - j < size), b * pool + pool - 1 <= i - size


def pooled_attention(q, k, v, scale, size, pool, cap, sink):
    """q [n, H, dim], k [n, G, dim], v [n, G, vdim].  ``pool`` None: a plain window; ``size`` None: causal."""
    n, H, _ = q.shape
    G = k.shape[1]
    if size is None:
        tok, blk = np.arange(n)[:, None] >= np.arange(n)[None, :], np.zeros((n, 0), dtype=bool)
        kb, vb = k[:0], v[:0]
    elif pool is None:
        tok, blk = pooled_window_masks(n, size, 1)[0], np.zeros((n, 0), dtype=bool)
        kb, vb = k[:0], v[:0]
    else:
        tok, blk = pooled_window_masks(n, size, pool)
        kb, vb = block_means(k, pool), block_means(v, pool)
    mask = np.concatenate([blk, tok], axis=1)
    out = np.zeros((n, H, v.shape[2]))
    for h in range(H):
        g = h // (H // G)
        s = softcap((q[:, h] @ np.concatenate([kb[:, g], k[:, g]]).T) * scale, cap)
        p = softmax_with_sink(s, mask, None if sink is None else sink[h])
        out[:, h] = p @ np.concatenate([vb[:, g], v[:, g]])
    return out.reshape(n, -1)


def left_attention(h, w, m, eps):
    n = h.shape[0]
    H, G, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rotate((h @ w["q"].T + w["q.b"]).reshape(n, H, dim), m.get("rot"), False)
    k = rotate((h @ w["k"].T + w["k.b"]).reshape(n, G, dim), m.get("rot"), False)
    v = (h @ w["v"].T + w["v.b"]).reshape(n, G, vdim)
    mask = m.get("mask") or {}
    o = pooled_attention(rms(q, eps), rms(k, eps), v, m["scale"], mask.get("size"), mask.get("pool"), m.get("softcap"),
                         w["sink"])
    return o @ w["o"].T


def retention(h, w, m, eps):
    n = h.shape[0]
    H, dim, vdim = m["heads"], m["dim"], m["vdim"]
    q = rotate((h @ w["q"].T).reshape(n, H, dim), m.get("rot"), False)
    k = rotate((h @ w["k"].T).reshape(n, H, dim), m.get("rot"), False) * dim ** -0.5
    v = (h @ w["v"].T).reshape(n, H, vdim)
    out = np.zeros((n, H, vdim))
    for x in range(H):
        S = np.zeros((dim, vdim))
        for t in range(n):
            S = m["decay"][x] * S + np.outer(k[t, x], v[t, x])
            out[t, x] = S.T @ q[t, x]
    return (rms(out, eps).reshape(n, -1) * silu(h @ w["g"].T)) @ w["o"].T


def parallel(h, w, m, eps):
    return (m["left_scale"] * left_attention(h, sub(w, "left."), m["left"], eps)
            + m["right_scale"] * retention(h, sub(w, "right."), m["right"], eps))


def squared_relu_unit(h, w):
    return np.maximum(h @ w["up"].T, 0.0) ** 2 @ w["down"].T


def gated_unit(h, w):
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def route(h, router, r):
    """(indices [n, top], weights [n, top]): softmax scores over all experts; the ``top`` largest inside the best
    ``keep`` groups (a group is as good as its best expert; the lower index wins a tie), renormalised, times the scale."""
    z = h @ router.T
    e = np.exp(z - z.max(axis=-1, keepdims=True))
    s = e / e.sum(axis=-1, keepdims=True)
    n, E = s.shape
    groups = r.get("groups") or {"count": 1, "keep": 1}
    gs = s.reshape(n, groups["count"], -1).max(axis=-1)
    best = np.argsort(-gs, axis=-1, kind="stable")[:, :groups["keep"]]
    ok = np.zeros((n, groups["count"]), dtype=bool)
    np.put_along_axis(ok, best, True, axis=-1)
    c = np.where(np.repeat(ok, E // groups["count"], axis=-1), s, -1.0)
    idx = np.argsort(-c, axis=-1, kind="stable")[:, :r["top"]]
    wt = np.take_along_axis(s, idx, axis=-1)
    return idx, wt / (wt.sum(axis=-1, keepdims=True) + 1e-20) * r.get("scale", 1.0)


def choice_margin(h, router, r):
    """How far, in router logits, each row is from another choice: the smaller of the gap between the worst kept group
    and the best group left out and the gap between the last chosen expert and the first one left out (inf if nothing
    is left out)."""
    z = h @ router.T
    n, E = z.shape
    groups = r.get("groups") or {"count": 1, "keep": 1}
    C, keep, top = groups["count"], groups["keep"], r["top"]
    gz = z.reshape(n, C, -1).max(axis=-1)
    order = np.argsort(-gz, axis=-1, kind="stable")
    gap = np.full(n, np.inf)
    if keep < C:
        s = np.take_along_axis(gz, order, axis=-1)
        gap = s[:, keep - 1] - s[:, keep]
    ok = np.zeros((n, C), dtype=bool)
    np.put_along_axis(ok, order[:, :keep], True, axis=-1)
    c = np.sort(np.where(np.repeat(ok, E // C, axis=-1), z, -np.inf), axis=-1)[:, ::-1]
    if top < keep * (E // C):
        gap = np.minimum(gap, c[:, top - 1] - c[:, top])
    return gap


def mixture(h, w, mlp, margins=None):
    r = mlp["router"]
    idx, wt = route(h, w["router"], r)
    if margins is not None:
        margins.append(choice_margin(h, w["router"], r))
    out = np.zeros_like(h)
    for e in range(r["experts"]):
        rows, col = np.nonzero(idx == e)
        if len(rows):
            out[rows] += wt[rows, col][:, None] * gated_unit(h[rows], sub(w, f"e{e}."))
    if mlp.get("shared"):
        out += gated_unit(h, sub(w, "shared."))
    return out


def gated_step(x, h, y, ls, rg, b):
    """The residual behind a sublayer: its output y, scaled a channel and gated by its input h."""
    return x + ls * sigmoid(h @ rg.T + b) * y


# ------------------------------------------------------------------- the model

def sub(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def forward(cfg, weights, tokens, return_layers=False, margins=None):
    """Logits [n, vocab] of a whole sequence (float64); with ``return_layers`` also the residual after every
    layer [layers, n, width]; ``margins`` (a list) gets every mixture's choice margins [n]."""
    eps = cfg["norm"]["eps"]
    W = {k: v.astype(np.float64) for k, v in weights.items()}
    x = W["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    after = []
    for i, L in enumerate(cfg["layers"]):
        w = sub(W, f"l{i}.")
        h = rms(x, eps) * w["norm1"]
        mixer = {"latent_attention": latent_attention, "parallel": parallel}[L["type"]]
        x = gated_step(x, h, mixer(h, sub(w, "mix."), L["mixer"], eps), w["ls1"], w["rg1"], w["rg1.b"])
        mlp = L.get("mlp")
        if mlp is not None:
            h = rms(x, eps) * w["norm2"]
            mw = sub(w, "mlp.")
            y = squared_relu_unit(h, mw) if mlp["kind"] == "dense" else mixture(h, mw, mlp, margins)
            x = gated_step(x, h, y, w["ls2"], w["rg2"], w["rg2.b"])
        after.append(x.copy())
    logits = (rms(x, eps) * W["final.norm"]) @ W["head"].T
    return (logits, np.stack(after)) if return_layers else logits


def load(model_dir):
    with open(os.path.join(model_dir, "config.json")) as f:
        cfg = json.load(f)
    return cfg, read_safetensors(os.path.join(model_dir, "model.safetensors"))


class PlainLadedra:
    """A model folder (or a configuration and tensors) with the whole-sequence forward pass above."""

    def __init__(self, model_dir=None, config=None, tensors=None):
        if model_dir is not None:
            self.cfg, self.w = load(model_dir)
        else:
            self.cfg, self.w = config, tensors

    def forward(self, tokens, layers_out=None, margins=None):
        logits, after = forward(self.cfg, self.w, tokens, True, margins)
        if layers_out is not None:
            layers_out.extend(after)
        return logits

    def logits(self, tokens):
        return self.forward(tokens)
