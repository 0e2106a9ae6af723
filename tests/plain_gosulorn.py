"""A plain, slow Gosulorn: whole sequences, no cache, one function for each mechanism.

Gosulorn is a decoder-only model whose residual is several streams.  A sublayer (mixer, then feed-forward) reads a
weighted sum of the streams through a layer norm without a shift; afterwards every stream is a weighted sum of all
the old streams plus its share of the sublayer's output.  Three mixers:

* ``gla``: linear attention whose state forgets with one data-dependent factor a key channel;
* ``delta``: the gated delta rule (the state is asked what it holds for the key, and the difference to the value is
  written), one data-dependent factor a head;
* ``parallel``: two mixers on the same input, their outputs weighed by two constants and added: windowed
  grouped-query softmax attention behind biases, short convolutions and a partial rotation; and the gated delta rule
  with one factor a key channel and low-rank factor and gate projections.

The feed-forward is a gated unit with the tanh form of gelu.  The output is the layer norm of the sum of the streams
times the embedding table.

This file shares no code with the package: it reads config.json and the safetensors file itself, with numpy only,
and runs in float64.
"""
from __future__ import annotations

import json
import math
import os
import struct

import numpy as np


def read_safetensors(path):
    """name -> numpy array (bfloat16 widened exactly; integer tables as they are)."""
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
        elif e["dtype"] == "I32":
            a = np.frombuffer(raw, dtype=np.int32)
        else:
            raise ValueError(f"{name}: dtype {e['dtype']}")
        out[name] = a.reshape(e["shape"]).copy()
    return out


# ------------------------------------------------------------------- mechanisms

def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def layer_norm(x, w, eps):
    d = x - np.mean(x, axis=-1, keepdims=True)
    return d / np.sqrt(np.mean(d * d, axis=-1, keepdims=True) + eps) * w


def unit_rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def unit_vector(x, eps=1e-6):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + eps)


def causal_conv(u, taps, before=None):
    """y[t, c] = sum_j taps[c, j] u[t - (K - 1) + j, c]: the last tap meets the current token; rows before the sequence
    count as zero, or are ``before`` ([K - 1, channels]: the inputs that came last)."""
    T, C = u.shape
    K = taps.shape[1]
    up = np.concatenate([np.zeros((K - 1, C)) if before is None else np.asarray(before, dtype=np.float64), u], 0)
    y = np.zeros((T, C))
    for j in range(K):
        y += up[j:j + T] * taps[:, j][None, :]
    return y


def rotate_half(x, dims, base, factor=1.0, first_pos=0):
    """x [T, heads, dim]: i < dims/2 is paired with i + dims/2, turned by p base^(-2i/dims) / factor; the rest passes."""
    T = x.shape[0]
    half = dims // 2
    f = np.power(float(base), -2.0 * np.arange(half) / dims) / factor
    a = (first_pos + np.arange(T))[:, None] * f[None, :]
    c, s = np.cos(a)[:, None, :], np.sin(a)[:, None, :]
    out = x.copy()
    u, v = x[..., :half], x[..., half:dims]
    out[..., :half] = u * c - v * s
    out[..., half:dims] = v * c + u * s
    return out


def windowed_attention(q, k, v, scale, window):
    """q [T, H, dim], k [T, G, dim], v [T, G, vdim]: row i sees j with 0 <= i - j < window (all j <= i if None)."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    o = np.zeros((T, H, v.shape[2]))
    for i in range(T):
        lo = 0 if window is None else max(0, i - int(window) + 1)
        for h in range(H):
            s = (k[lo:i + 1, h // per] @ q[i, h]) * scale
            p = np.exp(s - s.max())
            o[i, h] = (p / p.sum()) @ v[lo:i + 1, h // per]
    return o


def gated_scan(q, k, v, g, state=None):
    """Each row: the state's rows times their factors, plus the outer product of k and v; q reads.  q, k, g [T, H, dim], v [T, H, vdim]; o and the last state."""
    T, H, D = q.shape
    S = np.zeros((H, D, v.shape[2])) if state is None else np.array(state, dtype=np.float64)
    o = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        S = g[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hdp,hd->hp", S, q[t])
    return o, S


def delta_scan(q, k, v, g, beta, state=None):
    """Each row: F = g S, S' = F + k (beta (v - F^T k))^T; q reads S'.  q, k [T, H, dim], v [T, H, vdim], beta [T, H],
    g [T, H, dim] or [T, H, 1]; o and the last state."""
    T, H, D = q.shape
    S = np.zeros((H, D, v.shape[2])) if state is None else np.array(state, dtype=np.float64)
    o = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - np.einsum("hdp,hd->hp", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = np.einsum("hdp,hd->hp", S, q[t])
    return o, S


def conv_attention(h, w, m):
    """The left half of ``parallel``."""
    H, G, D, P = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q, k, v = (causal_conv(h @ w[n].T + w[n + ".b"], w[n + ".conv"]) for n in ("q", "k", "v"))
    q, k, v = q.reshape(T, H, D), k.reshape(T, G, D), v.reshape(T, G, P)
    rot = m.get("rot")
    if rot:
        factor = float(rot["scaling"]["factor"]) if rot.get("scaling") else 1.0
        q, k = (rotate_half(x, rot["dims"], rot["base"], factor) for x in (q, k))
    window = m["mask"]["size"] if m.get("mask") else None
    return windowed_attention(q, k, v, float(m["scale"]), window).reshape(T, H * P) @ w["o"].T + w["o.b"]


def delta_mixer(h, w, m, eps, per_channel):
    """The gated delta rule: ``per_channel`` with low-rank factors a key channel and a sigmoid gate (the right half of
    ``parallel``), else one factor a head and a silu gate."""
    H, G, D, P = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q, k, v = (silu(causal_conv(h @ w[n].T, w[n + ".conv"])) for n in ("q", "k", "v"))
    q = unit_vector(q.reshape(T, G, D)) * D ** -0.5
    k = unit_vector(k.reshape(T, G, D))
    q, k = (np.repeat(x, H // G, axis=1) for x in (q, k))
    beta = sigmoid(h @ w["b"].T)
    if per_channel:
        z = (softplus((h @ w["a1"].T) @ w["a2"].T + w["dt_bias"])).reshape(T, H, D)
        gate = sigmoid((h @ w["g1"].T) @ w["g2"].T)
    else:
        z = softplus(h @ w["a"].T + w["dt_bias"]).reshape(T, H, 1)
        gate = silu(h @ w["g"].T)
    g = np.exp(-np.exp(w["A_log"])[None, :, None] * z)
    o, _ = delta_scan(q, k, v.reshape(T, H, P), g, beta)
    return ((unit_rms(o, eps) * w["norm"]).reshape(T, H * P) * gate) @ w["o"].T


def gla_mixer(h, w, m, eps):
    H, D, P = m["heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = (h @ w["q"].T).reshape(T, H, D) * D ** -0.5
    k, v = (h @ w["k"].T).reshape(T, H, D), (h @ w["v"].T).reshape(T, H, P)
    z = ((h @ w["a1"].T) @ w["a2"].T + w["a2.b"]).reshape(T, H, D)
    o, _ = gated_scan(q, k, v, sigmoid(z) ** (1.0 / float(m["tau"])))
    return ((unit_rms(o, eps) * w["norm"]).reshape(T, H * P) * silu(h @ w["g"].T)) @ w["o"].T


def sub(w, prefix):
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def parallel_mixer(h, w, m, eps):
    return (float(m["left_scale"]) * conv_attention(h, sub(w, "left."), m["left"])
            + float(m["right_scale"]) * delta_mixer(h, sub(w, "right."), m["right"], eps, True))


def mixer(kind, h, w, m, eps):
    if kind == "parallel":
        return parallel_mixer(h, w, m, eps)
    if kind == "delta":
        return delta_mixer(h, w, m, eps, False)
    if kind == "gla":
        return gla_mixer(h, w, m, eps)
    raise ValueError(kind)


def gated_unit(h, w):
    return (gelu_tanh(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def streams_read(xs, w_in):
    """xs [T, s, d] -> [T, d]."""
    return np.einsum("tsd,s->td", xs, w_in)


def streams_write(xs, y, mix, out):
    """Every stream b from the old ones: out_b y + sum_a mix_ab x_a."""
    return np.einsum("nsd,st->ntd", xs, mix) + out[None, :, None] * y[:, None, :]


class PlainGosulorn:
    def __init__(self, model_dir=None, config=None, tensors=None):
        if model_dir is not None:
            with open(os.path.join(model_dir, "config.json")) as f:
                config = json.load(f)
            tensors = read_safetensors(os.path.join(model_dir, "model.safetensors"))
        self.cfg = config
        self.w = {k: np.asarray(v, dtype=np.float64) for k, v in tensors.items()}
        self.eps = float(config["norm"]["eps"])

    def forward(self, tokens, layers_out=None):
        """Logits [T, vocab] of a whole sequence; ``layers_out`` (a list) gets the sum of the streams after every layer."""
        cfg, w, eps = self.cfg, self.w, self.eps
        x = w["embed"][np.asarray(tokens)]
        xs = np.repeat(x[:, None, :], int(cfg["streams"]), axis=1)
        for i, L in enumerate(cfg["layers"]):
            while L.get("weights_of") is not None:
                i = int(L["weights_of"])
                L = cfg["layers"][i]
            p = f"l{i}."
            sublayers = [lambda h: mixer(L["type"], h, sub(w, p + "mix."), L["mixer"], eps)]
            if L.get("mlp") is not None:
                sublayers.append(lambda h: gated_unit(h, sub(w, p + "mlp.")))
            for n, f in enumerate(sublayers, 1):
                hc = sub(w, f"{p}hc{n}.")
                y = f(layer_norm(streams_read(xs, hc["in"]), w[f"{p}norm{n}"], eps))
                xs = streams_write(xs, y, hc["mix"], hc["out"])
            if layers_out is not None:
                layers_out.append(xs.sum(1))
        return layer_norm(xs.sum(1), w["final.norm"], eps) @ w["embed"].T
