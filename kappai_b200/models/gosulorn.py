"""Gosulorn: a decoder whose residual is several streams, with three kinds of linear-time mixer.

    x_1 .. x_s = embed[token]                                                    (``streams`` copies)
    a sublayer:  y = f(LN(sum_b in_b x_b)) ;  x'_b = out_b y + sum_a mix_ab x_a
    a layer:     its mixer, then its feed-forward, as such sublayers             (coefficients hc1, hc2; norms norm1, norm2)
    output:      logits = embed . LN(sum_b x_b)                                  (the table is the head; LN has no shift)

The mixers: ``gla`` (gated linear attention, one data-dependent factor a key channel; parts/gated.py), ``delta`` (the gated
delta rule, one factor a head, a silu gate; there too) and ``parallel`` (parts/parallel.py), the sum of two mixers on the
same input weighed by ``left_scale`` and ``right_scale``: on the left grouped-query attention over a sliding window with
biases, short convolutions on q, k and v and a rotation of a head's first dimensions with linearly scaled frequencies
(parts/attention.py), on the right the gated delta rule with one factor a key channel, low-rank projections for factors and
gate, and a sigmoid gate.  The feed-forward is a gated unit with the tanh form of gelu.

Where an entry says ``weights_of: j`` the schedule simply names layer j once more; what is remembered of a sequence belongs
to schedule entries, so the second run keeps its own.

This file is the only place that knows the design's ``config.json`` keys and tensor names: an
entry of ``layers`` holds ``type``, ``mixer`` and ``mlp`` (null where there is none), and tensors are named by the entry's
number, ``l0.`` on.  All sizes and constants come from the file or, for the low ranks, from the tensors' shapes;
what the design fixes (activations, the kinds of gate, norm and decay, the tied head) is written below.  ``mask``, ``rot`` and
``rot.scaling`` may be left out (every earlier key is read; nothing is rotated; frequencies as they are).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Optional

from ..config.schema import ConfigError, LayerSpec, ModelSpec, PartSpec, ScheduleEntry, TypedConfig, cfg
from ..config.registry import register_architecture

ARCHITECTURE = "Gosulorn"
FF_ACTIVATION = "gelu_tanh"
SOFTMAX_WEIGHTS = "float32"        # scores and weights are 32-bit, also where they meet the values
DEFAULT_MAX_POSITIONS = 131072     # the design itself sets no limit; an optional key ``max_positions`` overrides
MIXERS = ("parallel", "gla", "delta")


def _get(d: Any, key: str, where: str, typ=(int, float)):
    if not isinstance(d, dict) or key not in d or d[key] is None:
        raise ConfigError(f"config.json: missing required key '{where}.{key}'")
    v = d[key]
    if isinstance(v, bool) or not isinstance(v, typ):
        raise ConfigError(f"config key '{where}.{key}': unexpected value {v!r}")
    return v


def _int(d, key, where, least: int = 1) -> int:
    v = _get(d, key, where)
    if int(v) != v or int(v) < least:
        raise ConfigError(f"config key '{where}.{key}': expected an integer of at least {least}, got {v!r}")
    return int(v)


def _grouped(m, where: str) -> None:
    H, G = _int(m, "heads", where), _int(m, "kv_heads", where)
    _int(m, "dim", where), _int(m, "vdim", where), _int(m, "conv", where)
    if H % G:
        raise ConfigError(f"{where}: heads={H} must be a multiple of kv_heads={G}")


def _check_left(m, where: str) -> None:
    _grouped(m, where)
    _get(m, "scale", where)
    if m.get("mask") is not None:
        _int(m["mask"], "size", where + ".mask")
    rot = m.get("rot")
    if rot is not None:
        dims = _int(rot, "dims", where + ".rot")
        if not float(_get(rot, "base", where + ".rot")) > 0:
            raise ConfigError(f"{where}.rot.base must be positive")
        if dims < 2 or dims % 2 or dims > int(m["dim"]):
            raise ConfigError(f"{where}.rot.dims={dims} must be even and at most dim={m['dim']}")
        if rot.get("scaling") is not None and not float(_get(rot["scaling"], "factor", where + ".rot.scaling")) > 0:
            raise ConfigError(f"{where}.rot.scaling.factor must be positive")


@dataclass
class GosulornConfig(TypedConfig):
    vocab: int = cfg()
    width: int = cfg()
    layers: List[dict] = cfg()
    norm: dict = cfg()
    streams: int = cfg()
    max_positions: int = cfg(DEFAULT_MAX_POSITIONS)
    eos_token_id: Optional[int] = cfg(None)

    def validate(self) -> None:
        if self.vocab < 1 or self.width < 1:
            raise ConfigError("vocab and width must be positive")
        if not self.layers:
            raise ConfigError("layers must list at least one layer")
        if self.streams < 1:
            raise ConfigError("streams must be positive")
        if self.max_positions < 1:
            raise ConfigError("max_positions must be positive")
        self.eps = float(_get(self.norm, "eps", "norm"))
        if self.eps <= 0:
            raise ConfigError("norm.eps must be positive")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            if not isinstance(layer, dict):
                raise ConfigError(f"config key '{where}': expected an object")
            kind = _get(layer, "type", where, str)
            if kind not in MIXERS:
                raise ConfigError(f"config key '{where}.type'='{kind}': expected one of {', '.join(MIXERS)}")
            m, mw = _get(layer, "mixer", where, dict), where + ".mixer"
            if kind == "gla":
                for k in ("heads", "dim", "vdim"):
                    _int(m, k, mw)
                if not float(_get(m, "tau", mw)) > 0:
                    raise ConfigError(f"{mw}.tau must be positive")
            elif kind == "delta":
                _grouped(m, mw)
            else:
                _check_left(_get(m, "left", mw, dict), mw + ".left")
                _grouped(_get(m, "right", mw, dict), mw + ".right")
                _get(m, "left_scale", mw), _get(m, "right_scale", mw)
            mlp = layer.get("mlp")
            if mlp is not None:
                mk = _get(mlp, "kind", where + ".mlp", str)
                if mk != "dense":
                    raise ConfigError(f"config key '{where}.mlp.kind'='{mk}': this design has 'dense' feed-forwards only")
                _int(mlp, "ff", where + ".mlp")
        self.owner = [self._owner(i) for i in range(len(self.layers))]

    def _owner(self, i: int) -> int:
        """The layer whose tensors layer i runs with: itself, or where ``weights_of`` leads."""
        j, seen = i, set()
        while self.layers[j].get("weights_of") is not None:
            seen.add(j)
            where = f"layers[{j}]"
            k = _int(self.layers[j], "weights_of", where, 0)
            if k >= len(self.layers) or k in seen:
                raise ConfigError(f"{where}.weights_of={k} must name another layer that has tensors")
            for key in ("type", "mixer", "mlp"):
                if self.layers[k].get(key) != self.layers[j].get(key):
                    raise ConfigError(f"{where}.{key} differs from that of layer {k}, whose tensors it uses (weights_of)")
            j = k
        return j


def _delta_spec(c: GosulornConfig, m: Dict[str, Any], prefix: str, low_rank: bool, out_scale: float = 1.0) -> PartSpec:
    """The gated delta rule: with low-rank factors a key channel and gate (the right half of ``parallel``), or one factor a
    head and a whole gate projection (``delta``)."""
    rename = {"norm.weight": "norm", "beta_proj.weight": "b", "A_log": "A_log", "dt_bias": "dt_bias", "out_proj.weight": "o"}
    for n in ("q", "k", "v"):
        rename[f"{n}_proj.weight"], rename[f"{n}_conv.weight"] = n, f"{n}.conv"
    rename.update({"decay_down.weight": "a1", "decay_up.weight": "a2", "gate_down.weight": "g1", "gate_up.weight": "g2"} if low_rank
                  else {"decay_proj.weight": "a", "gate_proj.weight": "g"})
    return PartSpec(
        "gated_delta",
        {"hidden_size": c.width, "num_heads": int(m["heads"]), "num_qk_heads": int(m["kv_heads"]), "head_dim": int(m["dim"]),
         "value_dim": int(m["vdim"]), "conv_kernel": int(m["conv"]), "norm_eps": c.eps, "decay": "channel" if low_rank else "head",
         "gate": "sigmoid" if low_rank else "silu", "gate_rank": "low" if low_rank else "full", "out_scale": out_scale},
        prefix, rename=rename)


def _attention_spec(c: GosulornConfig, m: Dict[str, Any], prefix: str, out_scale: float) -> PartSpec:
    rot, position = m.get("rot"), None
    if rot is not None:
        scaling = rot.get("scaling")
        position = PartSpec("rope", {"rotary_dim": int(rot["dims"]), "theta": float(rot["base"]), "pairing": "neox",
                                     "scaling": None if scaling is None else {"factor": float(scaling["factor"])}})
    rename = {"out_proj.weight": "o", "out_proj.bias": "o.b"}
    for n in ("q", "k", "v"):
        rename[f"{n}_proj.weight"], rename[f"{n}_proj.bias"], rename[f"{n}_conv.weight"] = n, f"{n}.b", f"{n}.conv"
    return PartSpec(
        "attention",
        {"hidden_size": c.width, "num_heads": int(m["heads"]), "num_kv_heads": int(m["kv_heads"]), "head_dim": int(m["dim"]),
         "value_dim": int(m["vdim"]), "scale": float(m["scale"]), "qk_norm_eps": None, "bias": True, "conv_kernel": int(m["conv"]),
         "window": None if m.get("mask") is None else int(m["mask"]["size"]), "position": position,
         "softmax_weights": SOFTMAX_WEIGHTS, "out_scale": out_scale},
        prefix, rename=rename)


def _mixer_spec(c: GosulornConfig, layer: Dict[str, Any], prefix: str) -> PartSpec:
    m, kind = layer["mixer"], layer["type"]
    if kind == "delta":
        return _delta_spec(c, m, prefix, False)
    if kind == "gla":
        return PartSpec(
            "gated_linear",
            {"hidden_size": c.width, "num_heads": int(m["heads"]), "head_dim": int(m["dim"]), "value_dim": int(m["vdim"]),
             "tau": float(m["tau"]), "norm_eps": c.eps},
            prefix,
            rename={"q_proj.weight": "q", "k_proj.weight": "k", "v_proj.weight": "v", "gate_proj.weight": "g", "decay_down.weight": "a1",
                    "decay_up.weight": "a2", "decay_up.bias": "a2.b", "norm.weight": "norm", "out_proj.weight": "o"})
    return PartSpec("parallel", {"mixers": {"left": _attention_spec(c, m["left"], "", float(m["left_scale"])),
                                            "right": _delta_spec(c, m["right"], "", True, float(m["right_scale"]))}}, prefix)


def build_spec(c: GosulornConfig) -> ModelSpec:
    norm = lambda prefix, name: PartSpec("layernorm", {"size": c.width, "eps": c.eps}, prefix, rename={"weight": name})
    layers, ignored, number = [], [], {}
    for i in sorted(set(c.owner)):
        layer, p = c.layers[i], f"l{i}."
        mlp, ffn = layer.get("mlp"), None
        if mlp is not None:
            ffn = PartSpec("glu", {"hidden_size": c.width, "intermediate_size": int(mlp["ff"]), "activation": FF_ACTIVATION}, p + "mlp.",
                           rename={"gate_proj.weight": "gate", "up_proj.weight": "up", "down_proj.weight": "down"})
        else:
            ignored += [p + n for n in ("norm2", "hc2.in", "hc2.out", "hc2.mix")]     # of a feed-forward that the layer does not have
        number[i] = len(layers)
        layers.append(LayerSpec(mixer=_mixer_spec(c, layer, p + "mix."), ffn=ffn, mixer_norm=norm(p, "norm1"),
                                ffn_norm=norm(p, "norm2") if ffn is not None else None, block="streams_residual",
                                block_params={"streams": c.streams, "sublayers": 1 if ffn is None else 2}, block_prefix=p))
    spec = ModelSpec(
        architecture=ARCHITECTURE,
        hidden_size=c.width,
        vocab_size=c.vocab,
        max_positions=c.max_positions,
        embedding=PartSpec("embedding", {"vocab_size": c.vocab, "hidden_size": c.width, "scale": None}, "",
                           rename={"weight": "embed"}),
        layers=layers,
        schedule=[ScheduleEntry(number[j]) for j in c.owner],
        final_norm=norm("", "final.norm"),
        head=PartSpec("lm_head", {"vocab_size": c.vocab, "hidden_size": c.width, "tied": True}, ""),
        eos_token_id=c.eos_token_id,
        residual=PartSpec("streams", {"streams": c.streams, "hidden_size": c.width}),
        ignored_tensors=ignored,
    )
    spec.validate()
    return spec


register_architecture(ARCHITECTURE, GosulornConfig, build_spec)
