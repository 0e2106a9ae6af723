"""Ladedra: a decoder with scaled and gated sublayers, latent attention beside a windowed attention and a retention.

    x = embed[token] * embedding.scale
    a layer:   h = norm1(x) ;  x <- x + ls1 * sigmoid(Wg1 h + b1) * mixer(h)
               h = norm2(x) ;  x <- x + ls2 * sigmoid(Wg2 h + b2) * ff(h)                 (RMS norms with weights)
    output:    logits = head . norm(x)                                                    (a matrix of its own)

The mixers: ``latent_attention`` (parts/latent.py: one normed latent a token and a rotated key part that all heads share
are cached; interleaved pairs with YaRN frequencies; a sigmoid gate on the heads) and ``parallel`` (parts/parallel.py), the
sum of two mixers on the same input weighed by ``left_scale`` and ``right_scale``: on the left grouped-query attention with
biases on q, k and v, a norm without weights behind the rotation, soft-capped scores, a learned softmax sink, and a sliding
window behind which the means of blocks of ``mask.pool`` positions stay readable (parts/attention.py); on the right retention
with one constant decay a head (parts/lightning.py).  The feed-forward (parts/ffn.py) is an ungated unit with the square
of relu (``dense``) or a mixture of silu units (``moe``): softmax scores over all experts, the ``top`` largest inside the
best groups, renormalised and scaled, and a shared unit.

This file is the only place that knows the design's ``config.json`` keys and tensor names: an entry of ``layers`` holds
``type``, ``mixer`` and ``mlp`` (null where there is none), and tensors are named by the entry's number, ``l0.`` on.  All
sizes and constants come from there; what the design fixes (activations, the kinds of gate, norm and pairing) is
written below.  ``mask``, ``mask.pool``, ``softcap``, ``rot``, ``rot.scaling``, ``router.groups``, ``router.scale`` and an ``mlp``'s
``shared`` may be left out.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Optional

from ..config.schema import ConfigError, LayerSpec, ModelSpec, PartSpec, ScheduleEntry, TypedConfig, cfg
from ..config.registry import register_architecture

ARCHITECTURE = "Ladedra"
EXPERT_ACTIVATION = "silu"
DENSE_ACTIVATION = "relu_squared"
SOFTMAX_WEIGHTS = "float32"        # scores and weights are 32-bit, also where they meet the values
DEFAULT_MAX_POSITIONS = 131072     # the design itself sets no limit; an optional key ``max_positions`` overrides
MIXERS = ("latent_attention", "parallel")
YARN = ("factor", "original", "fast", "slow")


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


def _check_rot(rot, limit: int, where: str) -> None:
    if rot is None:
        return
    dims = _int(rot, "dims", where)
    if not float(_get(rot, "base", where)) > 0:
        raise ConfigError(f"{where}.base must be positive")
    if dims < 2 or dims % 2 or dims > limit:
        raise ConfigError(f"{where}.dims={dims} must be even and at most {limit}")
    if rot.get("scaling") is not None:
        for k in YARN:
            if not float(_get(rot["scaling"], k, where + ".scaling")) > 0:
                raise ConfigError(f"{where}.scaling.{k} must be positive")


def _check_left(m, where: str) -> None:
    H, G = _int(m, "heads", where), _int(m, "kv_heads", where)
    dim = _int(m, "dim", where)
    _int(m, "vdim", where), _get(m, "scale", where)
    if H % G:
        raise ConfigError(f"{where}: heads={H} must be a multiple of kv_heads={G}")
    if m.get("softcap") is not None and not float(_get(m, "softcap", where)) > 0:
        raise ConfigError(f"{where}.softcap must be positive")
    if m.get("mask") is not None:
        _int(m["mask"], "size", where + ".mask")
        if m["mask"].get("pool") is not None:
            _int(m["mask"], "pool", where + ".mask")
    _check_rot(m.get("rot"), dim, where + ".rot")


def _check_right(m, where: str) -> None:
    H, dim = _int(m, "heads", where), _int(m, "dim", where)
    _int(m, "vdim", where)
    decay = _get(m, "decay", where, list)
    if len(decay) != H:
        raise ConfigError(f"{where}.decay must list one number for each of the {H} heads")
    _check_rot(m.get("rot"), dim, where + ".rot")


@dataclass
class LadedraConfig(TypedConfig):
    vocab: int = cfg()
    width: int = cfg()
    layers: List[dict] = cfg()
    norm: dict = cfg()
    embedding: dict = cfg()
    max_positions: int = cfg(DEFAULT_MAX_POSITIONS)
    eos_token_id: Optional[int] = cfg(None)

    def validate(self) -> None:
        if self.vocab < 1 or self.width < 1:
            raise ConfigError("vocab and width must be positive")
        if not self.layers:
            raise ConfigError("layers must list at least one layer")
        if self.max_positions < 1:
            raise ConfigError("max_positions must be positive")
        self.eps = float(_get(self.norm, "eps", "norm"))
        if self.eps <= 0:
            raise ConfigError("norm.eps must be positive")
        self.embedding_scale = float(_get(self.embedding, "scale", "embedding"))
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            if not isinstance(layer, dict):
                raise ConfigError(f"config key '{where}': expected an object")
            kind = _get(layer, "type", where, str)
            if kind not in MIXERS:
                raise ConfigError(f"config key '{where}.type'='{kind}': expected one of {', '.join(MIXERS)}")
            m, mw = _get(layer, "mixer", where, dict), where + ".mixer"
            if kind == "latent_attention":
                for k in ("heads", "dim", "vdim", "kv_rank", "rot_dim"):
                    _int(m, k, mw)
                _get(m, "scale", mw)
                _check_rot(m.get("rot"), int(m["rot_dim"]), mw + ".rot")
            else:
                _check_left(_get(m, "left", mw, dict), mw + ".left")
                _check_right(_get(m, "right", mw, dict), mw + ".right")
                _get(m, "left_scale", mw), _get(m, "right_scale", mw)
            if layer.get("mlp") is not None:
                self._check_mlp(layer["mlp"], where + ".mlp")

    @staticmethod
    def _check_mlp(mlp, where: str) -> None:
        kind = _get(mlp, "kind", where, str)
        if kind == "dense":
            _int(mlp, "ff", where)
            return
        if kind != "moe":
            raise ConfigError(f"config key '{where}.kind'='{kind}': this design has 'dense' and 'moe' feed-forwards")
        _int(mlp.get("expert"), "ff", where + ".expert")
        r, rw = mlp.get("router"), where + ".router"
        E, top = _int(r, "experts", rw), _int(r, "top", rw)
        if top > E:
            raise ConfigError(f"{rw}: top={top} exceeds the {E} experts")
        if r.get("groups") is not None:
            count, keep = _int(r["groups"], "count", rw + ".groups"), _int(r["groups"], "keep", rw + ".groups")
            if E % count or keep > count or top > keep * (E // count):
                raise ConfigError(f"{rw}.groups: count={count} must divide the {E} experts, and keep={keep} groups must hold top={top} of them")
        if r.get("scale") is not None:
            _get(r, "scale", rw)
        if mlp.get("shared"):
            _int(mlp["shared"], "ff", where + ".shared")


def _rope(rot: Optional[Dict[str, Any]], pairing: str) -> Optional[PartSpec]:
    if rot is None:
        return None
    scaling = rot.get("scaling")
    return PartSpec("rope", {"rotary_dim": int(rot["dims"]), "theta": float(rot["base"]), "pairing": pairing,
                             "scaling": None if scaling is None else {k: float(scaling[k]) for k in YARN}})


def _left_spec(c: LadedraConfig, m: Dict[str, Any], out_scale: float) -> PartSpec:
    mask = m.get("mask") or {}
    rename = {"out_proj.weight": "o", "sink": "sink"}
    for n in ("q", "k", "v"):
        rename[f"{n}_proj.weight"], rename[f"{n}_proj.bias"] = n, f"{n}.b"
    return PartSpec(
        "attention",
        {"hidden_size": c.width, "num_heads": int(m["heads"]), "num_kv_heads": int(m["kv_heads"]), "head_dim": int(m["dim"]),
         "value_dim": int(m["vdim"]), "scale": float(m["scale"]), "qk_norm": "after_rotation", "qk_norm_eps": c.eps, "bias": "qkv",
         "window": None if not mask else int(mask["size"]), "pool": None if mask.get("pool") is None else int(mask["pool"]),
         "softcap": None if m.get("softcap") is None else float(m["softcap"]), "sink": "learned", "position": _rope(m.get("rot"), "neox"),
         "softmax_weights": SOFTMAX_WEIGHTS, "out_scale": out_scale},
        rename=rename)


def _right_spec(c: LadedraConfig, m: Dict[str, Any], out_scale: float) -> PartSpec:
    return PartSpec(
        "lightning",
        {"hidden_size": c.width, "num_heads": int(m["heads"]), "head_dim": int(m["dim"]), "value_dim": int(m["vdim"]),
         "decay": [float(a) for a in m["decay"]], "norm_eps": c.eps, "activation": None, "gate": "silu", "norm": "per_head",
         "position": _rope(m.get("rot"), "neox"), "k_scale": float(int(m["dim"])) ** -0.5, "out_scale": out_scale},
        rename={"q_proj.weight": "q", "k_proj.weight": "k", "v_proj.weight": "v", "gate_proj.weight": "g", "out_proj.weight": "o"})


def _mixer_spec(c: LadedraConfig, layer: Dict[str, Any], prefix: str) -> PartSpec:
    m = layer["mixer"]
    if layer["type"] == "latent_attention":
        return PartSpec(
            "latent_cache_attention",
            {"hidden_size": c.width, "num_heads": int(m["heads"]), "head_dim": int(m["dim"]), "rot_dim": int(m["rot_dim"]),
             "value_dim": int(m["vdim"]), "kv_rank": int(m["kv_rank"]), "scale": float(m["scale"]), "norm_eps": c.eps, "gate": "sigmoid",
             "position": _rope(m.get("rot"), "interleaved")},
            prefix,
            rename={"q_proj.weight": "q", "kv_down.weight": "dkv", "kv_norm.weight": "dkv.norm", "k_up.weight": "uk", "v_up.weight": "uv",
                    "gate_proj.weight": "g", "out_proj.weight": "o"})
    return PartSpec("parallel", {"mixers": {"left": _left_spec(c, m["left"], float(m["left_scale"])),
                                            "right": _right_spec(c, m["right"], float(m["right_scale"]))}}, prefix)


def _ffn_spec(c: LadedraConfig, mlp: Optional[Dict[str, Any]], prefix: str) -> Optional[PartSpec]:
    if mlp is None:
        return None
    if mlp["kind"] == "dense":
        return PartSpec("mlp", {"hidden_size": c.width, "intermediate_size": int(mlp["ff"]), "activation": DENSE_ACTIVATION}, prefix,
                        rename={"up_proj.weight": "up", "down_proj.weight": "down"})
    r = mlp["router"]
    E = int(r["experts"])
    rename = {"router.weight": "router"}
    for e in range(E):
        for n in ("gate", "up", "down"):
            rename[f"experts.{e}.{n}_proj.weight"] = f"e{e}.{n}"
    groups = r.get("groups")
    params = {"hidden_size": c.width, "expert_size": int(mlp["expert"]["ff"]), "num_experts": E, "top": int(r["top"]),
              "activation": EXPERT_ACTIVATION, "routing": "softmax_all", "correction": False, "renormalise": True,
              "router_scale": float(r["scale"]) if r.get("scale") is not None else 1.0,
              "groups": None if groups is None else {"count": int(groups["count"]), "keep": int(groups["keep"])}}
    if mlp.get("shared"):
        params.update(shared_size=int(mlp["shared"]["ff"]), shared_gate=None)
        rename.update({f"shared.{n}_proj.weight": f"shared.{n}" for n in ("gate", "up", "down")})
    return PartSpec("moe", params, prefix, rename=rename)


def build_spec(c: LadedraConfig) -> ModelSpec:
    norm = lambda prefix, name: PartSpec("rmsnorm", {"size": c.width, "eps": c.eps}, prefix, rename={"weight": name})
    layers, ignored = [], []
    for i, layer in enumerate(c.layers):
        p = f"l{i}."
        ffn = _ffn_spec(c, layer.get("mlp"), p + "mlp.")
        if ffn is None:
            ignored += [p + n for n in ("norm2", "ls2", "rg2", "rg2.b")]       # of a feed-forward that the layer does not have
        layers.append(LayerSpec(mixer=_mixer_spec(c, layer, p + "mix."), ffn=ffn, mixer_norm=norm(p, "norm1"),
                                ffn_norm=norm(p, "norm2") if ffn is not None else None, block="gated_residual",
                                block_params={"hidden_size": c.width, "sublayers": 1 if ffn is None else 2}, block_prefix=p,
                                block_rename={"rg1.weight": "rg1", "rg1.bias": "rg1.b", "rg2.weight": "rg2", "rg2.bias": "rg2.b"}))
    spec = ModelSpec(
        architecture=ARCHITECTURE,
        hidden_size=c.width,
        vocab_size=c.vocab,
        max_positions=c.max_positions,
        embedding=PartSpec("embedding", {"vocab_size": c.vocab, "hidden_size": c.width, "scale": c.embedding_scale}, "",
                           rename={"weight": "embed"}),
        layers=layers,
        schedule=[ScheduleEntry(i) for i in range(len(layers))],
        final_norm=norm("", "final.norm"),
        head=PartSpec("lm_head", {"vocab_size": c.vocab, "hidden_size": c.width, "tied": False}, "", rename={"weight": "head"}),
        eos_token_id=c.eos_token_id,
        ignored_tensors=ignored,
    )
    spec.validate()
    return spec


register_architecture(ARCHITECTURE, LadedraConfig, build_spec)
