"""Typed configuration of Futezen: a decoder whose layers put an RMS norm on both sides of every sublayer (weights
stored around zero), mix along the sequence by attention over a cached low-rank latent with low-rank queries, by
grouped-query attention, or by a state-space recurrence, and feed forward densely or through routed experts
beside a gated shared one; a stretch of layers may run several times.

``config.json`` keys: ``architecture`` ("Futezen"), ``vocab``, ``width``, ``norm.eps``, ``loop`` (``start``, ``stop``,
``times``: layers start .. stop-1 run ``times`` times in a row with the same weights, every pass with a cache or state
of its own; absent: every layer once) and ``layers``, a list whose entries give ``type``, ``mixer`` (its sizes and
constants) and ``mlp`` (a feed-forward, or null).

* ``latent_attention``: ``heads``, ``dim``, ``rot_dim``, ``vdim``, ``q_rank``, ``kv_rank``, ``scale``, ``rot`` =
  ``base`` (all of the ``rot_dim`` part turns, neighbours pair up).
* ``attention``: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``rot`` = ``base``, ``dims`` (halves pair up;
  absent: nothing turns).
* ``mamba2``: ``heads``, ``vdim``, ``state``, ``groups``, ``conv`` (taps), ``norm_groups``.
* ``mlp``: ``{"kind": "dense", "ff"}`` (relu on the gate) or ``{"kind": "moe", "expert": {"ff"}, "router":
  {"experts", "top"}, "shared": {"ff"} or absent}`` (experts without a gate, the square of relu).

Tensor names: ``embed``, ``final.norm``; layer i: ``l<i>.norm1``, ``norm1b``, ``norm2``, ``norm2b``;
``mix.{dq,dq.norm,uq,dkv,dkv.norm,uk,uv,o}``, ``mix.{q,k,v,o}`` or ``mix.{in,conv,conv.b,dt_bias,A_log,D,norm,o}``;
``mlp.{gate,up,down}``, or ``mlp.router``, ``mlp.router.b``, ``mlp.e<j>.{up,down}``, ``mlp.shared.{up,down,sg}``.  The
head is the embedding table.  The file states no context limit: the engine's page pool is the only one.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, Mapping, Optional, Tuple

from .lfm2 import ConfigError
from .spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

UNBOUNDED_POSITIONS = 1 << 24
NAME = "Futezen"


def _need(mapping: Any, keys, where: str) -> None:
    if not isinstance(mapping, Mapping):
        raise ConfigError(f"{NAME} config.json: {where} must be an object")
    missing = [key for key in keys if mapping.get(key) is None]
    if missing:
        raise ConfigError(f"{NAME} config.json: {where} is missing " + ", ".join(missing))


def _positive(mapping: Mapping[str, Any], keys, where: str) -> None:
    for key in keys:
        if not float(mapping[key]) > 0:
            raise ConfigError(f"{NAME} config.json: {where}: {key} must be positive")


def _sizes(mapping: Any, keys, where: str) -> None:
    _need(mapping, keys, where)
    _positive(mapping, keys, where)


def _multiple(mapping, of: str, by: str, where: str) -> None:
    if int(mapping[of]) % int(mapping[by]):
        raise ConfigError(f"{NAME} config.json: {where}: {of} must be a multiple of {by}")


def _check_rot(rot, where: str, dims_at_most: int) -> None:
    _need(rot, ("base", "dims"), where)
    _positive(rot, ("base",), where)
    if int(rot["dims"]) % 2 or not 0 <= int(rot["dims"]) <= dims_at_most:
        raise ConfigError(f"{NAME} config.json: {where}: dims must be even and at most {dims_at_most}")


def _rope(rot, pairing: str) -> PartSpec:
    if rot is None or int(rot["dims"]) <= 0:
        return PartSpec("no_position")
    return PartSpec("rope", {"theta": float(rot["base"]), "rotary_dim": int(rot["dims"]), "pairing": pairing})


@dataclass(frozen=True)
class FutezenConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[Mapping[str, Any], ...]          # as config.json gives them, checked
    loop: Optional[Tuple[int, int, int]] = None    # (start, stop, times)
    architectures: Tuple[str, ...] = (NAME,)
    extra: Mapping[str, Any] = field(default_factory=dict, compare=False)

    # ------------------------------------------------------------------ reading / writing
    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "FutezenConfig":
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
            cls._check_mixer(layer["type"], layer["mixer"], where)
            if layer.get("mlp") is not None:
                cls._check_mlp(layer["mlp"], where)
            layers.append(layer)
        loop = raw.get("loop")
        if loop is not None:
            _need(loop, ("start", "stop", "times"), "'loop'")
            start, stop, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
            if not 0 <= start <= stop <= len(layers) or times < 1:
                raise ConfigError(f"{NAME} config.json: 'loop' must have 0 <= start <= stop <= {len(layers)} and "
                                  "times >= 1")
            loop = (start, stop, times)
        known = {"architecture", "architectures", "vocab", "width", "norm", "layers", "loop"}
        return cls(vocab=int(raw["vocab"]), width=int(raw["width"]), norm_eps=float(raw["norm"]["eps"]),
                   layers=tuple(layers), loop=loop, extra={k: v for k, v in raw.items() if k not in known})

    @staticmethod
    def _check_mixer(kind: str, mixer, where: str) -> None:
        inside = f"{where}'s mixer"
        if kind == "latent_attention":
            _need(mixer, ("rot_dim", "scale", "rot"), inside)
            _sizes(mixer, ("heads", "dim", "vdim", "q_rank", "kv_rank"), inside)
            if int(mixer["rot_dim"]) < 0 or int(mixer["rot_dim"]) % 2:
                raise ConfigError(f"{NAME} config.json: {where}: rot_dim must be even and not negative")
            _sizes(mixer["rot"], ("base",), f"{inside}.rot")
        elif kind == "attention":
            _need(mixer, ("scale",), inside)
            _sizes(mixer, ("heads", "kv_heads", "dim", "vdim"), inside)
            _multiple(mixer, "heads", "kv_heads", where)
            if mixer.get("rot") is not None:
                _check_rot(mixer["rot"], f"{inside}.rot", int(mixer["dim"]))
        elif kind == "mamba2":
            _sizes(mixer, ("heads", "vdim", "state", "groups", "conv", "norm_groups"), inside)
            _multiple(mixer, "heads", "groups", where)
            if int(mixer["heads"]) * int(mixer["vdim"]) % int(mixer["norm_groups"]):
                raise ConfigError(f"{NAME} config.json: {where}: heads * vdim must be a multiple of norm_groups")
        else:
            raise ConfigError(f"{NAME} config.json: {where} has the unknown type {kind!r} "
                              "(known: latent_attention, attention, mamba2)")

    @staticmethod
    def _check_mlp(mlp, where: str) -> None:
        inside = f"{where}'s mlp"
        _need(mlp, ("kind",), inside)
        if mlp["kind"] == "dense":
            _sizes(mlp, ("ff",), inside)
        elif mlp["kind"] == "moe":
            _need(mlp, ("expert", "router"), inside)
            _sizes(mlp["expert"], ("ff",), f"{inside}.expert")
            _sizes(mlp["router"], ("experts", "top"), f"{inside}.router")
            if int(mlp["router"]["top"]) > int(mlp["router"]["experts"]):
                raise ConfigError(f"{NAME} config.json: {where}: top exceeds the number of experts")
            if mlp.get("shared") is not None:
                _sizes(mlp["shared"], ("ff",), f"{inside}.shared")
        else:
            raise ConfigError(f"{NAME} config.json: {where} has the unknown feed-forward {mlp['kind']!r} "
                              "(known: dense, moe)")

    def to_dict(self) -> dict:
        out = {"architecture": self.architectures[0], "vocab": self.vocab, "width": self.width,
               "norm": {"eps": self.norm_eps}, "layers": copy.deepcopy(list(self.layers))}
        if self.loop is not None:
            out["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        out.update(self.extra)
        return out

    # ------------------------------------------------------------------ the model in parts
    def runs(self):
        """The layer index of every execution, in order."""
        n = len(self.layers)
        if self.loop is None:
            return list(range(n))
        start, stop, times = self.loop
        return list(range(start)) + list(range(start, stop)) * times + list(range(stop, n))

    def _latent(self, m, prefix: str) -> PartSpec:
        return PartSpec(
            "latent_attention",
            {"hidden_size": self.width, "num_heads": int(m["heads"]), "dim": int(m["dim"]),
             "rot_dim": int(m["rot_dim"]), "vdim": int(m["vdim"]), "kv_rank": int(m["kv_rank"]),
             "q_rank": int(m["q_rank"]), "scale": float(m["scale"]), "eps": self.norm_eps, "sink": False,
             "position": _rope({"base": m["rot"]["base"], "dims": m["rot_dim"]}, "interleaved")},
            {"dq": prefix + "dq", "dq_norm": prefix + "dq.norm", "uq": prefix + "uq", "dkv": prefix + "dkv",
             "dkv_norm": prefix + "dkv.norm", "uk": prefix + "uk", "uv": prefix + "uv", "o": prefix + "o"})

    def _attention(self, m, prefix: str) -> PartSpec:
        return PartSpec(
            "gqa_attention",
            {"hidden_size": self.width, "num_heads": int(m["heads"]), "num_kv_heads": int(m["kv_heads"]),
             "head_dim": int(m["dim"]), "value_dim": int(m["vdim"]), "scale": float(m["scale"]),
             "qk_norm_eps": None, "position": _rope(m.get("rot"), "half_split")},
            {role: prefix + role for role in ("q", "k", "v", "o")})

    def _state_space(self, m, prefix: str) -> PartSpec:
        return PartSpec(
            "state_space",
            {"hidden_size": self.width, "num_heads": int(m["heads"]), "vdim": int(m["vdim"]), "state": int(m["state"]),
             "groups": int(m["groups"]), "taps": int(m["conv"]), "norm_groups": int(m["norm_groups"]),
             "eps": self.norm_eps},
            {"in": prefix + "in", "conv": prefix + "conv", "conv_bias": prefix + "conv.b",
             "dt_bias": prefix + "dt_bias", "a_log": prefix + "A_log", "skip": prefix + "D", "norm": prefix + "norm",
             "o": prefix + "o"})

    def _feed_forward(self, mlp, prefix: str) -> PartSpec:
        if mlp["kind"] == "dense":
            return PartSpec("swiglu", {"hidden_size": self.width, "ffn_dim": int(mlp["ff"]), "activation": "relu"},
                            {role: prefix + role for role in ("gate", "up", "down")})
        experts = int(mlp["router"]["experts"])
        params = {"hidden_size": self.width, "ffn_dim": int(mlp["expert"]["ff"]), "experts": experts,
                  "top": int(mlp["router"]["top"]), "activation": "relu_squared", "gated": False,
                  "scores": "softmax_chosen"}
        tensors = {"router": prefix + "router", "correction": prefix + "router.b"}
        for j in range(experts):
            for role in ("up", "down"):
                tensors[f"{role}{j}"] = f"{prefix}e{j}.{role}"
        if mlp.get("shared") is not None:
            params.update(shared_ffn_dim=int(mlp["shared"]["ff"]), shared_scaled=True)
            tensors.update(shared_up=prefix + "shared.up", shared_down=prefix + "shared.down",
                           shared_scale=prefix + "shared.sg")
        return PartSpec("routed_experts", params, tensors)

    def model_spec(self) -> ModelSpec:
        def norm(name: str) -> PartSpec:
            return PartSpec("rmsnorm", {"size": self.width, "eps": self.norm_eps, "offset": 1.0}, {"weight": name})

        mixers = {"latent_attention": self._latent, "attention": self._attention, "mamba2": self._state_space}
        layers = []
        for index, layer in enumerate(self.layers):
            prefix = f"l{index}."
            parts = {"mixer_norm": norm(prefix + "norm1"),
                     "mixer": mixers[layer["type"]](layer["mixer"], prefix + "mix."),
                     "mixer_out_norm": norm(prefix + "norm1b")}
            if layer.get("mlp") is not None:
                parts["ffn_norm"] = norm(prefix + "norm2")
                parts["feed_forward"] = self._feed_forward(layer["mlp"], prefix + "mlp.")
                parts["ffn_out_norm"] = norm(prefix + "norm2b")
            layers.append(LayerSpec("sandwich_residual", parts=parts))
        spec = ModelSpec(
            architecture=self.architectures[0], hidden_size=self.width, vocab_size=self.vocab,
            max_positions=UNBOUNDED_POSITIONS, embedding_tensor="embed", final_norm=norm("final.norm"),
            head_tensor=None, layers=tuple(layers), schedule=tuple(ScheduleEntry(i) for i in self.runs()))
        spec.validate()
        return spec
