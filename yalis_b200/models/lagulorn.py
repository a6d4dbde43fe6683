"""Lagulorn as an architecture of this engine: a pre-norm decoder whose residual stream is kept in several copies.

Token rows are scaled as they enter; the stream then exists in ``streams`` copies, of which every sub-layer reads a
weighted sum and to all of which it writes, its result times ``residual_mult`` (without ``streams``: the plain residual
sum, times that constant).  The norm is RMS with a weight stored around zero.  A layer's mixer is one of

* ``lightning``  a matrix per head with a fixed decay: S_t = d_h S_(t-1) + k_t v_t^T, o_t = S_t^T q_t, with q, k, v through
                 silu; all heads of the read-out are normed together and gated by a sigmoid;
* ``attention``  differential attention: two maps per head over the same values, each a softmax over a window; their
                 weighted difference is normed per head.  Queries and keys are normed per head and map, nothing is
                 rotated.

The feed-forward is dense (``gelu`` in its erf form), a mixture of clamped gated experts, or absent.  The experts' router
chooses by corrected softmax scores among the best groups of neighbouring outputs and weighs by the scores themselves; its
last outputs are identity experts.  A layer with ``weights_of`` runs another layer's tensors with a cache or state of its own.

``config.json`` gives every size and every constant that models of the design may differ in; this file holds what the
design fixes.  Like every architecture here the model is described as data.
"""

from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Dict, List, Mapping, Optional, Tuple

from yalis_b200.config.registry import ConfigError, register_architecture
from yalis_b200.config.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

ARCHITECTURE_NAME = "Lagulorn"
MAX_POSITION = 1 << 20          # nothing in the design bounds a sequence; block tables are sized by the cache pool
LAYER_TYPES = ("lightning", "attention")
CLAMP_ALPHA, CLAMP_SHIFT = 1.702, 1.0     # experts: g sigmoid(CLAMP_ALPHA g) (u + CLAMP_SHIFT)


@dataclass(frozen=True)
class LagulornConfig:
    width: int
    vocab: int
    streams: Optional[int]                    # copies of the residual stream (None: a plain stream)
    norm_eps: float
    embedding_scale: float
    residual_mult: float
    layers: Tuple[Mapping[str, Any], ...]     # validated copies of the config's layer entries

    @property
    def architecture(self) -> str:
        return ARCHITECTURE_NAME

    def owner(self, i: int) -> int:
        """The layer whose tensors layer ``i`` runs."""
        while self.layers[i].get("weights_of") is not None:
            i = self.layers[i]["weights_of"]
        return i


def _int(d, key: str, where: str, least: int = 1) -> int:
    v = d.get(key) if isinstance(d, Mapping) else None
    if isinstance(v, bool) or not isinstance(v, int) or v < least:
        raise ConfigError(f"{where}: `{key}` must be an integer of at least {least}, got {v!r}")
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


def _lightning(m, where: str) -> Dict[str, Any]:
    out: Dict[str, Any] = {k: _int(m, k, where) for k in ("heads", "dim", "vdim")}
    decay = m.get("decay")
    if not isinstance(decay, (list, tuple)) or len(decay) != out["heads"] or any(isinstance(d, bool) or not isinstance(d, (int, float)) for d in decay):
        raise ConfigError(f"{where}: `decay` must hold a number for each of the {out['heads']} heads, got {decay!r}")
    out["decay"] = [float(d) for d in decay]
    return out


def _attention(m, where: str) -> Dict[str, Any]:
    out: Dict[str, Any] = {k: _int(m, k, where) for k in ("heads", "kv_heads", "dim", "vdim")}
    if out["heads"] % out["kv_heads"]:
        raise ConfigError(f"{where}: heads {out['heads']} is not a multiple of kv_heads {out['kv_heads']}")
    out.update({k: _num(m, k, where) for k in ("scale", "diff")})
    if m.get("mask") is not None:
        out["mask"] = {"size": _int(m["mask"], "size", where + ".mask")}
    return out


def _mlp(mlp, where: str) -> Optional[Dict[str, Any]]:
    if mlp is None:
        return None
    kind = mlp.get("kind") if isinstance(mlp, Mapping) else mlp
    if kind == "dense":
        return {"kind": "dense", "ff": _int(mlp, "ff", where)}
    if kind != "moe":
        raise ConfigError(f"{where}: kind {kind!r} is not supported (dense, moe, or null)")
    r = mlp.get("router")
    router: Dict[str, Any] = {k: _int(r, k, where + ".router") for k in ("experts", "top")}
    outputs = router["experts"]
    if r.get("identity") is not None:
        router["identity"] = _int(r, "identity", where + ".router", least=0)
        outputs += router["identity"]
    room = outputs
    if r.get("groups") is not None:
        g = router["groups"] = {k: _int(r["groups"], k, where + ".router.groups") for k in ("count", "keep")}
        if outputs % g["count"] or g["keep"] > g["count"]:
            raise ConfigError(f"{where}.router: {outputs} outputs do not form {g['count']} equal groups of which {g['keep']} are kept")
        room = outputs // g["count"] * g["keep"]
    if router["top"] > room:
        raise ConfigError(f"{where}.router: top {router['top']} is more than the {room} outputs to choose from")
    return {"kind": "moe", "router": router, "expert": {"ff": _int(mlp.get("expert"), "ff", where + ".expert"),
                                                        "limit": _positive(mlp.get("expert"), "limit", where + ".expert")}}


def _check_layer(i: int, layer) -> Dict[str, Any]:
    where = f"layers[{i}]"
    kind = layer.get("type") if isinstance(layer, Mapping) else None
    if kind not in LAYER_TYPES:
        raise ConfigError(f"{where}: type {kind!r} is not one of {', '.join(LAYER_TYPES)}")
    if not isinstance(layer.get("mixer"), Mapping):
        raise ConfigError(f"{where}: `mixer` must be an object")
    mixer = _lightning(layer["mixer"], where) if kind == "lightning" else _attention(layer["mixer"], where)
    out = {"type": kind, "mixer": mixer, "mlp": _mlp(layer.get("mlp"), where + ".mlp")}
    if layer.get("weights_of") is not None:
        out["weights_of"] = _int(layer, "weights_of", where, least=0)
    return out


def _check_sharing(layers: List[Dict[str, Any]]) -> None:
    """Every chain of ``weights_of`` ends at a layer with tensors, whose entry is the same."""
    for i, layer in enumerate(layers):
        at, seen = i, {i}
        while layers[at].get("weights_of") is not None:
            at = layers[at]["weights_of"]
            if at >= len(layers) or at in seen:
                raise ConfigError(f"layers[{i}]: weights_of leads to {at}, which is no layer with tensors of its own")
            seen.add(at)
        for key in ("type", "mixer", "mlp"):
            if layer[key] != layers[at][key]:
                raise ConfigError(f"layers[{i}]: `{key}` is not that of layer {at}, whose tensors it uses")


class LagulornArchitecture:
    name = ARCHITECTURE_NAME

    @staticmethod
    def parse_config(raw: Dict[str, Any]) -> LagulornConfig:
        layers = raw.get("layers")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config.json lacks `layers`")
        checked = [_check_layer(i, l) for i, l in enumerate(layers)]
        _check_sharing(checked)
        emb = raw.get("embedding")
        return LagulornConfig(
            width=_int(raw, "width", "config"), vocab=_int(raw, "vocab", "config"),
            streams=_int(raw, "streams", "config") if raw.get("streams") is not None else None,
            norm_eps=_positive(raw.get("norm"), "eps", "norm"),
            embedding_scale=_num(emb, "scale", "embedding") if emb is not None and emb.get("scale") is not None else 1.0,
            residual_mult=_num(raw, "residual_mult", "config") if raw.get("residual_mult") is not None else 1.0,
            layers=tuple(checked))

    @staticmethod
    def config_to_dict(c: LagulornConfig) -> Dict[str, Any]:
        d = {"architecture": ARCHITECTURE_NAME, "embedding": {"scale": c.embedding_scale},
             "layers": copy.deepcopy([dict(l) for l in c.layers]), "norm": {"eps": c.norm_eps}, "residual_mult": c.residual_mult,
             "vocab": c.vocab, "width": c.width}
        if c.streams is not None:
            d["streams"] = c.streams
        return d

    @staticmethod
    def _norm(c: LagulornConfig) -> PartSpec:
        return PartSpec("rms_norm", {"size": c.width, "eps": c.norm_eps, "one_plus": True})

    @staticmethod
    def _connection(c: LagulornConfig) -> PartSpec:
        if c.streams is None:
            return PartSpec("scaled_sum", {"hidden_size": c.width, "learned": False, "factor": c.residual_mult})
        return PartSpec("hyper_connection", {"hidden_size": c.width, "copies": c.streams, "mixing": True, "factor": c.residual_mult})

    @staticmethod
    def _mixer(c: LagulornConfig, kind: str, m: Mapping[str, Any]):
        """The mixer's part and the tensor names of its parameters."""
        if kind == "lightning":
            part = PartSpec("retention", {
                "hidden_size": c.width, "heads": m["heads"], "dim": m["dim"], "vdim": m["vdim"], "decay": m["decay"],
                "rotary": None, "eps": c.norm_eps, "activation": "silu", "norm": "all", "gate": "sigmoid"})
            return part, {f"mixer.{p}_proj": f"mix.{p}" for p in "qkvgo"} | {"mixer.norm": "mix.norm"}
        part = PartSpec("general_attention", {
            "hidden_size": c.width, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"],
            "v_head_dim": m["vdim"], "bias": False, "qk_norm_eps": c.norm_eps, "rotary": None, "scale": m["scale"],
            "window": m["mask"]["size"] if m.get("mask") else None, "difference": {"offset": m["diff"], "eps": c.norm_eps}})
        names = {f"mixer.{p}_proj": f"mix.{p}" for p in "qkvo"} | {f"mixer.{p}_norm": f"mix.{p}.norm" for p in "qk"}
        return part, names | {f"mixer.{p}": f"mix.{p}" for p in ("lq1", "lk1", "lq2", "lk2")}

    @staticmethod
    def _feed_forward(c: LagulornConfig, mlp: Mapping[str, Any]):
        if mlp["kind"] == "dense":
            part = PartSpec("dense", {"hidden_size": c.width, "intermediate_size": mlp["ff"], "activation": "gelu_erf"})
            return part, {f"feed_forward.{p}_proj": f"mlp.{p}" for p in ("up", "down")}
        r = mlp["router"]
        part = PartSpec("routed_experts", {
            "hidden_size": c.width, "experts": r["experts"], "top": r["top"], "expert_size": mlp["expert"]["ff"], "gated": True,
            "activation": "clamped", "limit": mlp["expert"]["limit"], "alpha": CLAMP_ALPHA, "shift": CLAMP_SHIFT,
            "shared_size": None, "renorm": False, "correction": True, "groups": r.get("groups"), "identity": r.get("identity", 0)})
        names = {"feed_forward.router": "mlp.router", "feed_forward.correction": "mlp.correction"}
        for e in range(r["experts"]):
            names.update({f"feed_forward.expert_{e}_{p}": f"mlp.e{e}.{p}" for p in ("gate", "up", "down")})
        return part, names

    @classmethod
    def _layer(cls, c: LagulornConfig, i: int) -> LayerSpec:
        layer = c.layers[i]
        mixer, names = cls._mixer(c, layer["type"], layer["mixer"])
        parts = {"norm_1": cls._norm(c), "mixer": mixer, "connection_1": cls._connection(c)}
        sublayers = [1]
        if layer["mlp"] is not None:
            sublayers.append(2)
            parts["feed_forward"], ff_names = cls._feed_forward(c, layer["mlp"])
            parts["norm_2"], parts["connection_2"] = cls._norm(c), cls._connection(c)
            names.update(ff_names)
        for q in sublayers:
            names[f"norm_{q}.weight"] = f"norm{q}"
            if c.streams is not None:
                names.update({f"connection_{q}.{p}": f"hc{q}.{p}" for p in ("in", "out", "mix")})
        return LayerSpec(block=PartSpec("pre_norm_connected"), parts=parts, weight_prefix=f"l{i}.", weight_names=names)

    @classmethod
    def model_spec(cls, c: LagulornConfig) -> ModelSpec:
        owners = [i for i in range(len(c.layers)) if c.owner(i) == i]
        place = {i: at for at, i in enumerate(owners)}
        return ModelSpec(
            architecture=ARCHITECTURE_NAME, hidden_size=c.width, vocab_size=c.vocab, max_position=MAX_POSITION,
            layers=tuple(cls._layer(c, i) for i in owners),
            schedule=tuple(ScheduleEntry(place[c.owner(i)]) for i in range(len(c.layers))),
            final_norm=cls._norm(c), embedding_name="embed", head_name="head", final_norm_names={"weight": "final.norm"},
            embedding_scale=c.embedding_scale, stream_copies=c.streams)


register_architecture(ARCHITECTURE_NAME, LagulornArchitecture, replace=True)
