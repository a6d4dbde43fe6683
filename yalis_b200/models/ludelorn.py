"""Ludelorn as an architecture of this engine: a pre-norm decoder whose norms have one learned number each, whose
sub-layers' results are multiplied by a learned vector before they join the stream, and whose layers have one of three
mixers:

* ``parallel``     windowed attention (a norm on every head of q and k, half-split rotation with YaRN frequencies, a
                   sigmoid gate per element) beside a selective state space with a scalar decay per head (Mamba-2); each
                   result is normed over the model's width, and half their sum is the mixer's;
* ``attention``    a norm over all heads of q (of k) at once, interleaved rotation, a window and beside it the pooled
                   blocks of ``mask.pool`` positions that lie before it, a gate per element;
* ``attention_2``  the values are the raw keys, heads are brought to unit root mean square, no rotation: a learned bias
                   per distance bucket and head; a window, a learned sink, a gate per head.

The feed-forward is dense with biases and the tanh form of gelu, or absent.  Token rows are scaled as they enter the
stream.  ``config.json`` gives every size and constant but one: the number of distance buckets, which
``sizes_from_tensors`` reads from the checkpoint's header (a configuration written by this package carries it as
``buckets``).  Like every architecture here the model is described as data.
"""

from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Dict, Mapping, Optional, Tuple

from yalis_b200.config.registry import ConfigError, register_architecture
from yalis_b200.config.spec import LayerSpec, ModelSpec, PartSpec, default_schedule

ARCHITECTURE_NAME = "Ludelorn"
MAX_POSITION = 1 << 20          # nothing in the design bounds a sequence; block tables are sized by the cache pool
LAYER_TYPES = ("parallel", "attention", "attention_2")
SIDES_FACTOR = 0.5              # the parallel mixer's result is this times the sum of its two normed sides


@dataclass(frozen=True)
class LudelornConfig:
    width: int
    vocab: int
    norm_eps: float
    embedding_scale: float
    layers: Tuple[Mapping[str, Any], ...]     # validated copies of the config's layer entries

    @property
    def architecture(self) -> str:
        return ARCHITECTURE_NAME


def _int(d, key: str, where: str) -> int:
    v = d.get(key) if isinstance(d, Mapping) else None
    if isinstance(v, bool) or not isinstance(v, int) or v <= 0:
        raise ConfigError(f"{where}: `{key}` must be a positive integer, got {v!r}")
    return v


def _num(d, key: str, where: str) -> float:
    v = d.get(key) if isinstance(d, Mapping) else None
    if isinstance(v, bool) or not isinstance(v, (int, float)):
        raise ConfigError(f"{where}: `{key}` must be a number, got {v!r}")
    return float(v)


def _positive(d, key: str, where: str) -> float:
    v = _num(d, key, where)
    if v <= 0:
        raise ConfigError(f"{where}: `{key}` must be positive, got {v!r}")
    return v


def _heads(m, where: str) -> Dict[str, Any]:
    out: Dict[str, Any] = {k: _int(m, k, where) for k in ("heads", "kv_heads", "dim", "vdim")}
    if out["heads"] % out["kv_heads"]:
        raise ConfigError(f"{where}: heads {out['heads']} is not a multiple of kv_heads {out['kv_heads']}")
    out["scale"] = _num(m, "scale", where)
    return out


def _rot(m, dim: int, where: str) -> Optional[Dict[str, Any]]:
    rot = m.get("rot")
    if rot is None:
        return None
    where += ".rot"
    dims, base = _int(rot, "dims", where), _num(rot, "base", where)
    if dims % 2 or dims > dim or base <= 1.0:
        raise ConfigError(f"{where}: dims {dims} must be even and at most {dim}, base above 1")
    out: Dict[str, Any] = {"dims": dims, "base": base}
    if rot.get("scaling") is not None:
        out["scaling"] = {k: _positive(rot["scaling"], k, where + ".scaling") for k in ("factor", "original", "fast", "slow")}
    return out


def _mask(m, where: str) -> Optional[Dict[str, int]]:
    mask = m.get("mask")
    if mask is None:
        return None
    out = {"size": _int(mask, "size", where + ".mask")}
    if mask.get("pool") is not None:
        out["pool"] = _int(mask, "pool", where + ".mask")
    return out


def _attention(m, where: str) -> Dict[str, Any]:
    out = _heads(m, where)
    for key, value in (("mask", _mask(m, where)), ("rot", _rot(m, out["dim"], where))):
        if value is not None:
            out[key] = value
    return out


def _biased(m, where: str) -> Dict[str, Any]:
    out = _heads(m, where)
    if out["vdim"] != out["dim"]:
        raise ConfigError(f"{where}: vdim {out['vdim']} must equal dim {out['dim']}: the values are the keys")
    mask = _mask(m, where)
    if mask is not None:
        out["mask"] = mask
    out["bias_max"] = m.get("bias_max")
    _num(m, "bias_max", where)
    if m.get("buckets") is None:
        raise ConfigError(f"{where}: `buckets` is not given (a model folder gives it by the shape of its tensors)")
    out["buckets"] = _int(m, "buckets", where)
    if out["buckets"] % 2 or out["bias_max"] <= out["buckets"] // 2:
        raise ConfigError(f"{where}: the number of buckets, {out['buckets']}, must be even and half of it below bias_max {out['bias_max']}")
    return out


def _state_space(m, where: str) -> Dict[str, Any]:
    out = {k: _int(m, k, where) for k in ("heads", "vdim", "state", "groups", "norm_groups", "conv")}
    if out["heads"] % out["groups"]:
        raise ConfigError(f"{where}: heads {out['heads']} is not a multiple of groups {out['groups']}")
    if out["heads"] * out["vdim"] % out["norm_groups"]:
        raise ConfigError(f"{where}: {out['heads'] * out['vdim']} columns do not divide into norm_groups {out['norm_groups']}")
    return out


def _check_layer(i: int, layer) -> Dict[str, Any]:
    where = f"layers[{i}]"
    kind = layer.get("type") if isinstance(layer, Mapping) else None
    if kind not in LAYER_TYPES:
        raise ConfigError(f"{where}: type {kind!r} is not one of {', '.join(LAYER_TYPES)}")
    m = layer.get("mixer")
    if not isinstance(m, Mapping):
        raise ConfigError(f"{where}: `mixer` must be an object")
    if kind == "parallel":
        for side in ("left", "right"):
            if not isinstance(m.get(side), Mapping):
                raise ConfigError(f"{where}: a parallel mixer needs `{side}`")
        mixer: Dict[str, Any] = {"left": _attention(m["left"], where + ".left"), "right": _state_space(m["right"], where + ".right")}
    else:
        mixer = _attention(m, where) if kind == "attention" else _biased(m, where)
    mlp = layer.get("mlp")
    if mlp is not None:
        if not isinstance(mlp, Mapping) or mlp.get("kind") != "dense":
            raise ConfigError(f"{where}: mlp kind {mlp.get('kind') if isinstance(mlp, Mapping) else mlp!r} is not supported (dense, or null)")
        mlp = {"kind": "dense", "ff": _int(mlp, "ff", where + ".mlp")}
    return {"type": kind, "mixer": mixer, "mlp": mlp}


class LudelornArchitecture:
    name = ARCHITECTURE_NAME

    @staticmethod
    def sizes_from_tensors(raw: Dict[str, Any], shapes: Mapping[str, Tuple[int, ...]]) -> Dict[str, Any]:
        """The configuration with the size that only a tensor's shape gives filled in."""
        raw = copy.deepcopy(raw)
        for i, layer in enumerate(raw.get("layers") or []):
            if isinstance(layer, dict) and layer.get("type") == "attention_2" and isinstance(layer.get("mixer"), dict):
                shape = shapes.get(f"l{i}.mix.rel")
                if shape is not None and len(shape) == 2:
                    layer["mixer"]["buckets"] = int(shape[0])
        return raw

    @staticmethod
    def parse_config(raw: Dict[str, Any]) -> LudelornConfig:
        layers = raw.get("layers")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config.json lacks `layers`")
        scale = _num(raw.get("embedding"), "scale", "embedding") if raw.get("embedding") is not None else 1.0
        return LudelornConfig(width=_int(raw, "width", "config"), vocab=_int(raw, "vocab", "config"),
                              norm_eps=_positive(raw.get("norm"), "eps", "norm"), embedding_scale=scale,
                              layers=tuple(_check_layer(i, l) for i, l in enumerate(layers)))

    @staticmethod
    def config_to_dict(c: LudelornConfig) -> Dict[str, Any]:
        return {"architecture": ARCHITECTURE_NAME, "embedding": {"scale": c.embedding_scale},
                "layers": copy.deepcopy([dict(l) for l in c.layers]), "norm": {"eps": c.norm_eps}, "vocab": c.vocab, "width": c.width}

    @classmethod
    def _norm(cls, c: LudelornConfig) -> PartSpec:
        return PartSpec("rms_norm", {"size": c.width, "eps": c.norm_eps, "scalar": True})

    @staticmethod
    def _attention_params(c: LudelornConfig, m: Mapping[str, Any]) -> Dict[str, Any]:
        mask = m.get("mask") or {}
        return {"hidden_size": c.width, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"],
                "v_head_dim": m["vdim"], "bias": False, "qk_norm_eps": c.norm_eps, "scale": m["scale"],
                "window": mask.get("size"), "pool": mask.get("pool")}

    @staticmethod
    def _rotary(m: Mapping[str, Any], layout: str) -> Optional[Dict[str, Any]]:
        rot = m.get("rot")
        if rot is None:
            return None
        sc = rot.get("scaling")
        return {"dims": rot["dims"], "theta": rot["base"], "layout": layout, "scaling": None if sc is None else {"kind": "yarn", **sc}}

    @classmethod
    def _mixer(cls, c: LudelornConfig, kind: str, m: Mapping[str, Any]):
        """The mixer's part and the tensor names of its parameters."""
        def named(prefix: str, under: str, *locals_: str, **others: str) -> Dict[str, str]:
            return {f"{prefix}{n}_proj": f"{under}{n}" for n in locals_} | {f"{prefix}{k}": f"{under}{v}" for k, v in others.items()}

        if kind == "attention":
            part = PartSpec("general_attention", {**cls._attention_params(c, m), "qk_norm_over": "all", "gate": True,
                                                  "rotary": cls._rotary(m, "interleaved")})
            return part, named("mixer.", "mix.", "q", "k", "v", "g", "o", q_norm="q.norm", k_norm="k.norm")
        if kind == "attention_2":
            part = PartSpec("general_attention", {
                **cls._attention_params(c, m), "qk_norm_weight": False, "values_from_keys": True, "rotary": None,
                "distance_bias": {"buckets": m["buckets"], "max": m["bias_max"]}, "sink": "learned", "gate": "head"})
            return part, named("mixer.", "mix.", "q", "k", "g", "o", rel="rel", sink="sink")
        left, right = m["left"], m["right"]
        attention = PartSpec("general_attention", {**cls._attention_params(c, left), "gate": True, "rotary": cls._rotary(left, "half")})
        state = PartSpec("state_space", {
            "hidden_size": c.width, "heads": right["heads"], "vdim": right["vdim"], "state": right["state"],
            "groups": right["groups"], "norm_groups": right["norm_groups"], "conv": right["conv"], "eps": c.norm_eps})
        part = PartSpec("sum_of_mixers", {"mixers": {"left": attention, "right": state}, "norm_eps": c.norm_eps,
                                          "factor": SIDES_FACTOR})
        names = named("mixer.left.", "mix.left.", "q", "k", "v", "g", "o", q_norm="q.norm", k_norm="k.norm", out_norm="out")
        names.update(named("mixer.right.", "mix.right.", "in", "o", conv="conv", conv_bias="conv.b", dt_bias="dt_bias", A_log="A_log",
                           D="D", norm="norm", out_norm="out"))
        return part, names

    @classmethod
    def _layer(cls, c: LudelornConfig, i: int, layer: Mapping[str, Any]) -> LayerSpec:
        mixer, names = cls._mixer(c, layer["type"], layer["mixer"])
        scaled = PartSpec("scaled_sum", {"hidden_size": c.width})
        parts = {"norm_1": cls._norm(c), "mixer": mixer, "connection_1": scaled}
        names.update({"norm_1.weight": "norm1", "connection_1.scale": "ls1"})
        if layer["mlp"] is not None:
            parts.update({"norm_2": cls._norm(c), "connection_2": scaled, "feed_forward": PartSpec("dense", {
                "hidden_size": c.width, "intermediate_size": layer["mlp"]["ff"], "activation": "gelu_tanh", "bias": True})})
            names.update({"norm_2.weight": "norm2", "connection_2.scale": "ls2", "feed_forward.up_proj": "mlp.up",
                          "feed_forward.up_bias": "mlp.up.b", "feed_forward.down_proj": "mlp.down",
                          "feed_forward.down_bias": "mlp.down.b"})
        return LayerSpec(block=PartSpec("pre_norm_connected"), parts=parts, weight_prefix=f"l{i}.", weight_names=names)

    @classmethod
    def model_spec(cls, c: LudelornConfig) -> ModelSpec:
        return ModelSpec(
            architecture=ARCHITECTURE_NAME, hidden_size=c.width, vocab_size=c.vocab, max_position=MAX_POSITION,
            layers=tuple(cls._layer(c, i, layer) for i, layer in enumerate(c.layers)), schedule=default_schedule(len(c.layers)),
            final_norm=cls._norm(c), embedding_name="embed", head_name="head", final_norm_names={"weight": "final.norm"},
            embedding_scale=c.embedding_scale)


register_architecture(ARCHITECTURE_NAME, LudelornArchitecture, replace=True)
