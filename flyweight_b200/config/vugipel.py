"""Typed configuration of Vugipel: a pre-norm decoder whose layers mix along the sequence with a minGRU, or with
a windowed softmax attention beside a retention, and whose feed-forwards are experts behind a sigmoid router.

``config.json`` keys: ``architecture`` ("Vugipel"), ``vocab``, ``width``, ``norm.eps`` and ``layers``, a list whose
entries give ``type`` ("mingru" | "parallel"), ``mixer`` (its sizes and constants) and ``mlp`` (a feed-forward,
or null).

* ``mingru``: ``width`` (channels of the recurrence).
* ``parallel``: ``left_scale``, ``right_scale`` and two mixers.  ``left``: ``heads``, ``kv_heads``, ``dim``,
  ``vdim``, ``scale``, ``softcap`` (absent: scores are not capped), ``mask`` = ``size``, ``keep_first`` (a sliding
  window and the first positions that stay visible; absent: every earlier key) and ``rot`` = ``base``, ``dims``
  (of queries and keys; values turn over all of ``vdim`` with the same base; absent: nothing turns).
  ``right``: ``heads``, ``dim``, ``vdim``, ``decay`` (one number per head).
* ``mlp``: ``{"kind": "moe", "expert": {"ff"}, "router": {"experts", "top"}}``.

Tensor names: ``embed``, ``head``, ``final.norm``; layer i: ``l<i>.norm1``, ``norm2`` (stored around zero);
``mix.{z,z.b,x,x.b,g,o}`` for minGRU; ``mix.left.{q,q.b,k,k.b,v,v.b,q.norm,k.norm,temp,o,o.b}`` and
``mix.right.{q,k,v,g,o}`` for the pair; ``mlp.router``, ``mlp.e<j>.{gate,up,down}``.  The file states no context
limit: the engine's page pool is the only one.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, Mapping, Tuple

from .lfm2 import ConfigError
from .spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

UNBOUNDED_POSITIONS = 1 << 24
NAME = "Vugipel"


def _need(mapping: Any, keys, where: str) -> None:
    if not isinstance(mapping, Mapping):
        raise ConfigError(f"{NAME} config.json: {where} must be an object")
    missing = [key for key in keys if mapping.get(key) is None]
    if missing:
        raise ConfigError(f"{NAME} config.json: {where} is missing " + ", ".join(missing))


def _positive(mapping: Mapping[str, Any], keys, where: str) -> None:
    for key in keys:
        if int(mapping[key]) <= 0:
            raise ConfigError(f"{NAME} config.json: {where}: {key} must be positive")


def _check_left(left, where: str) -> None:
    _need(left, ("heads", "kv_heads", "dim", "vdim", "scale"), where)
    _positive(left, ("heads", "kv_heads", "dim", "vdim"), where)
    if int(left["heads"]) % int(left["kv_heads"]):
        raise ConfigError(f"{NAME} config.json: {where}: heads must be a multiple of kv_heads")
    rot = left.get("rot")
    if rot is not None:
        _need(rot, ("base", "dims"), f"{where}.rot")
        if int(rot["dims"]) % 2 or not 0 <= int(rot["dims"]) <= int(left["dim"]):
            raise ConfigError(f"{NAME} config.json: {where}: rot.dims must be even and at most dim")
        if int(left["vdim"]) % 2:
            raise ConfigError(f"{NAME} config.json: {where}: rotated values need an even vdim")
    mask = left.get("mask")
    if mask is not None:
        _need(mask, ("size",), f"{where}.mask")
        _positive(mask, ("size",), f"{where}.mask")
        if int(mask.get("keep_first") or 0) < 0:
            raise ConfigError(f"{NAME} config.json: {where}: mask.keep_first must not be negative")
    if float(left.get("softcap") or 0.0) < 0:
        raise ConfigError(f"{NAME} config.json: {where}: softcap must not be negative")


def _check_right(right, where: str) -> None:
    _need(right, ("heads", "dim", "vdim", "decay"), where)
    _positive(right, ("heads", "dim", "vdim"), where)
    if len(right["decay"]) != int(right["heads"]):
        raise ConfigError(f"{NAME} config.json: {where}: one decay per head")


def _check_mlp(mlp, where: str) -> None:
    _need(mlp, ("kind",), where)
    if mlp["kind"] != "moe":
        raise ConfigError(f"{NAME} config.json: {where}: unknown feed-forward {mlp['kind']!r} (known: moe)")
    _need(mlp, ("expert", "router"), where)
    _need(mlp["expert"], ("ff",), f"{where}.expert")
    _need(mlp["router"], ("experts", "top"), f"{where}.router")
    _positive(mlp["expert"], ("ff",), f"{where}.expert")
    _positive(mlp["router"], ("experts", "top"), f"{where}.router")
    if int(mlp["router"]["top"]) > int(mlp["router"]["experts"]):
        raise ConfigError(f"{NAME} config.json: {where}: top exceeds the number of experts")


@dataclass(frozen=True)
class VugipelConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[Mapping[str, Any], ...]          # as config.json gives them, checked
    architectures: Tuple[str, ...] = (NAME,)
    extra: Mapping[str, Any] = field(default_factory=dict, compare=False)

    # ------------------------------------------------------------------ reading / writing
    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "VugipelConfig":
        _need(raw, ("vocab", "width", "norm", "layers"), "the top level")
        _need(raw["norm"], ("eps",), "'norm'")
        _positive(raw, ("vocab", "width"), "the top level")
        if not isinstance(raw["layers"], (list, tuple)) or not raw["layers"]:
            raise ConfigError(f"{NAME} config.json: 'layers' must be a list with at least one layer")
        layers = []
        for index, layer in enumerate(raw["layers"]):
            where = f"layer {index}"
            _need(layer, ("type", "mixer"), where)
            layer = copy.deepcopy(dict(layer))
            mixer = layer["mixer"]
            if layer["type"] == "mingru":
                _need(mixer, ("width",), f"{where}'s mixer")
                _positive(mixer, ("width",), f"{where}'s mixer")
            elif layer["type"] == "parallel":
                _need(mixer, ("left", "right", "left_scale", "right_scale"), f"{where}'s mixer")
                _check_left(mixer["left"], f"{where}'s mixer.left")
                _check_right(mixer["right"], f"{where}'s mixer.right")
            else:
                raise ConfigError(f"{NAME} config.json: {where} has the unknown type {layer['type']!r} "
                                  "(known: mingru, parallel)")
            if layer.get("mlp") is not None:
                _check_mlp(layer["mlp"], f"{where}'s mlp")
            layers.append(layer)
        known = {"architecture", "architectures", "vocab", "width", "norm", "layers"}
        return cls(vocab=int(raw["vocab"]), width=int(raw["width"]), norm_eps=float(raw["norm"]["eps"]),
                   layers=tuple(layers), extra={k: v for k, v in raw.items() if k not in known})

    def to_dict(self) -> dict:
        out = {"architecture": self.architectures[0], "vocab": self.vocab, "width": self.width,
               "norm": {"eps": self.norm_eps}, "layers": copy.deepcopy(list(self.layers))}
        out.update(self.extra)
        return out

    # ------------------------------------------------------------------ the model in parts
    def _left(self, m, prefix: str) -> PartSpec:
        rot, mask = m.get("rot"), m.get("mask") or {}
        # (angles of the values exist wherever there is a rotation, also one of no key channels)
        position = (PartSpec("rope", {"theta": float(rot["base"]), "rotary_dim": int(rot["dims"]),
                                      "pairing": "interleaved"}) if rot is not None else PartSpec("no_position"))
        window = int(mask.get("size") or 0)
        return PartSpec(
            "gqa_attention",
            {"hidden_size": self.width, "num_heads": int(m["heads"]), "num_kv_heads": int(m["kv_heads"]),
             "head_dim": int(m["dim"]), "value_dim": int(m["vdim"]), "scale": float(m["scale"]),
             "qk_norm_eps": self.norm_eps, "position": position, "window": window,
             "keep_first": int(mask.get("keep_first") or 0) if window else 0,
             "softcap": float(m.get("softcap") or 0.0), "bias": True, "temp": True,
             "turned_values": rot is not None},
            {"q": prefix + "q", "k": prefix + "k", "v": prefix + "v", "o": prefix + "o", "q_b": prefix + "q.b",
             "k_b": prefix + "k.b", "v_b": prefix + "v.b", "o_b": prefix + "o.b", "q_norm": prefix + "q.norm",
             "k_norm": prefix + "k.norm", "temp": prefix + "temp"})

    def _right(self, m, prefix: str) -> PartSpec:
        return PartSpec(
            "decayed_linear_attention",
            {"hidden_size": self.width, "num_heads": int(m["heads"]), "dim": int(m["dim"]), "vdim": int(m["vdim"]),
             "decay": tuple(float(x) for x in m["decay"]), "eps": self.norm_eps, "activation": None,
             "k_scale": float(m["dim"]) ** -0.5, "norm": "head", "gate": "silu"},
            {name: prefix + name for name in ("q", "k", "v", "g", "o")})

    def _experts(self, mlp, prefix: str) -> PartSpec:
        E = int(mlp["router"]["experts"])
        tensors = {"router": prefix + "router"}
        for j in range(E):
            for role in ("gate", "up", "down"):
                tensors[f"{role}{j}"] = f"{prefix}e{j}.{role}"
        return PartSpec(
            "routed_experts",
            {"hidden_size": self.width, "ffn_dim": int(mlp["expert"]["ff"]), "experts": E,
             "top": int(mlp["router"]["top"]), "activation": "silu", "scores": "sigmoid", "corrected": False,
             "weights_on": "input"},
            tensors)

    def model_spec(self) -> ModelSpec:
        W, eps = self.width, self.norm_eps

        def norm(name: str) -> PartSpec:
            return PartSpec("rmsnorm", {"size": W, "eps": eps, "offset": 1.0}, {"weight": name})

        layers, unused = [], []
        for index, layer in enumerate(self.layers):
            prefix = f"l{index}."
            m = layer["mixer"]
            if layer["type"] == "mingru":
                p = prefix + "mix."
                mixer = PartSpec("mingru", {"hidden_size": W, "width": int(m["width"])},
                                 {"z": p + "z", "z_b": p + "z.b", "x": p + "x", "x_b": p + "x.b", "g": p + "g",
                                  "o": p + "o"})
            else:
                mixer = PartSpec(
                    "mixer_pair",
                    {"hidden_size": W, "combine": "scaled", "left_scale": float(m["left_scale"]),
                     "right_scale": float(m["right_scale"]), "left": self._left(m["left"], prefix + "mix.left."),
                     "right": self._right(m["right"], prefix + "mix.right.")})
            parts = {"mixer_norm": norm(prefix + "norm1"), "mixer": mixer}
            if layer.get("mlp") is not None:
                parts["ffn_norm"] = norm(prefix + "norm2")
                parts["feed_forward"] = self._experts(layer["mlp"], prefix + "mlp.")
            else:
                unused.append(prefix + "norm2")
            layers.append(LayerSpec("prenorm_residual", parts=parts))
        spec = ModelSpec(
            architecture=self.architectures[0], hidden_size=W, vocab_size=self.vocab,
            max_positions=UNBOUNDED_POSITIONS, embedding_tensor="embed", final_norm=norm("final.norm"),
            head_tensor="head", layers=tuple(layers),
            schedule=tuple(ScheduleEntry(i) for i in range(len(self.layers))), unused_tensors=tuple(unused))
        spec.validate()
        return spec
