"""Typed configuration of the Vononex decoder, read from config.json.

Keys: `architecture` ("Vononex"), `vocab`, `width`, `norm.eps`, `postln_alpha` and `layers`, a list whose entries have
`type`, the mixer's sizes under `mixer`, and `mlp` (null or {`kind`: `dense`, `ff`}).

    parallel   left:  heads, kv_heads, dim, vdim, scale, rot {base, dims}           (attention)
               right: heads, dim, vdim, rot {base, dims}, decay (one number a head)  (linear attention with a fixed decay)
               and left_scale, right_scale beside them
    mingru     width                                                                (a gated elementwise recurrence)

The design, as the plan states it: the norm comes behind the sum, x becomes the RMS norm of alpha x + sublayer(x), with
the same alpha everywhere and the sublayers reading x itself.  The mixer `parallel` is a weighted sum of two mixers that
read the same rows.  The left one is grouped-query attention with biases on all four projections, queries and keys normed
over their whole rows (all heads together) in front of the rotation, a learned factor per head on the scores, and values
that are turned by their own position before they are cached, each head's output being turned back by the query's.  The
right one keeps a matrix of state per head that decays by a constant of the head; queries and keys are rotated, the heads'
outputs are divided by their root mean square, gated and projected.  The mixer `mingru` moves every channel of its state
towards a candidate by a gate, both made from the present token alone, and gates the state on its way out.  The
feed-forward is a gated product with the tanh form of gelu and biases.  The model's norm and a head of its own.
Tensor names: `embed`, `final.norm`, `head`, and per layer i `l<i>.norm1`, `.norm2`, `.mix.*` (`.mix.left.*`,
`.mix.right.*`), `.mlp.*`; a bias has its matrix's name with `.b` added.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Dict, List

from .plan import LayerSpec, ModelPlan, PartSpec, SubPart, default_schedule
from .registry import ConfigError, register_architecture

_TYPES = ("parallel", "mingru")
_MLPS = ("dense",)


def _integer(where: str, raw, key: str, least: int = 1) -> int:
    v = raw.get(key) if isinstance(raw, dict) else None
    if isinstance(v, bool) or not isinstance(v, (int, float)) or int(v) != v:
        raise ConfigError(f"config.json (Vononex): {where}`{key}` must be an integer, got {v!r}")
    if int(v) < least:
        raise ConfigError(f"config.json (Vononex): {where}`{key}` must be at least {least}, got {v}")
    return int(v)


def _number(where: str, raw, key: str) -> float:
    v = raw.get(key) if isinstance(raw, dict) else None
    if isinstance(v, bool) or not isinstance(v, (int, float)):
        raise ConfigError(f"config.json (Vononex): {where}`{key}` must be a number, got {v!r}")
    return float(v)


def _rotation(where: str, m: dict) -> None:
    dims = _integer(where + "rot.", m.get("rot"), "dims", least=2)
    if dims % 2 or dims > m["dim"]:
        raise ConfigError(f"Vononex config: {where}rot.dims {dims} must be even and at most dim {m['dim']}")
    if not _number(where + "rot.", m["rot"], "base") > 0:
        raise ConfigError(f"Vononex config: {where}rot.base must be positive")


@register_architecture("Vononex", "vononex")
@dataclass
class VononexConfig:
    vocab: int
    width: int
    layers: List[Dict[str, Any]]
    postln_alpha: float
    norm_eps: float = 1e-6
    max_positions: int = 1 << 20            # nothing in the design bounds a sequence

    architecture = "Vononex"
    model_type = "vononex"

    @property
    def vocab_size(self) -> int:            # the name generic callers use
        return self.vocab

    # ------------------------------------------------------------------ reading
    @classmethod
    def from_dict(cls, raw: dict) -> "VononexConfig":
        for key in ("vocab", "width", "layers", "postln_alpha"):
            if raw.get(key) is None:
                raise ConfigError(f"config.json (Vononex): missing key `{key}`")
        if not isinstance(raw["layers"], list) or not raw["layers"]:
            raise ConfigError("config.json (Vononex): `layers` must be a non-empty list")
        cfg = cls(
            vocab=_integer("", raw, "vocab"), width=_integer("", raw, "width"), layers=copy.deepcopy(raw["layers"]),
            postln_alpha=_number("", raw, "postln_alpha"), norm_eps=float((raw.get("norm") or {}).get("eps", 1e-6)),
            max_positions=_integer("", raw, "max_positions") if raw.get("max_positions") is not None else 1 << 20)
        cfg.validate()
        return cfg

    def validate(self) -> None:
        if not self.norm_eps > 0:
            raise ConfigError(f"Vononex config: norm.eps must be positive, got {self.norm_eps}")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]."
            kind = layer.get("type") if isinstance(layer, dict) else None
            if kind not in _TYPES:
                raise ConfigError(f"Vononex config: {where}type must be one of {_TYPES}, got {kind!r}")
            m = layer.get("mixer")
            if not isinstance(m, dict):
                raise ConfigError(f"Vononex config: {where}mixer is missing")
            if kind == "mingru":
                _integer(where + "mixer.", m, "width")
            else:
                self._validate_parallel(m, where + "mixer.")
            mlp = layer.get("mlp")
            if mlp is not None:
                if not isinstance(mlp, dict) or mlp.get("kind") not in _MLPS:
                    raise ConfigError(f"Vononex config: {where}mlp.kind must be one of {_MLPS}")
                _integer(where + "mlp.", mlp, "ff")

    @staticmethod
    def _validate_parallel(m: dict, where: str) -> None:
        left, right = m.get("left"), m.get("right")
        if not isinstance(left, dict) or not isinstance(right, dict):
            raise ConfigError(f"Vononex config: {where}left and {where}right are needed")
        lw, rw = where + "left.", where + "right."
        for key in ("heads", "kv_heads", "dim", "vdim"):
            _integer(lw, left, key)
        if left["heads"] % left["kv_heads"]:
            raise ConfigError(f"Vononex config: {lw}heads {left['heads']} are not a multiple of kv_heads {left['kv_heads']}")
        for key in ("dim", "vdim"):
            if left[key] % 2 or left[key] > 256:
                raise ConfigError(f"Vononex config: {lw}{key} {left[key]} must be even and at most 256")
        if not _number(lw, left, "scale") > 0:
            raise ConfigError(f"Vononex config: {lw}scale must be positive")
        _rotation(lw, left)
        for key in ("heads", "dim", "vdim"):
            _integer(rw, right, key)
        if right["dim"] > 512:
            raise ConfigError(f"Vononex config: {rw}dim {right['dim']} is beyond the scan kernel's 512")
        _rotation(rw, right)
        decay = right.get("decay")
        if not isinstance(decay, list) or len(decay) != right["heads"] or not all(
                isinstance(v, (int, float)) and not isinstance(v, bool) for v in decay):
            raise ConfigError(f"Vononex config: {rw}decay must list one number for each of the {right['heads']} heads")
        _number(where, m, "left_scale")
        _number(where, m, "right_scale")

    # ------------------------------------------------------------------ writing
    def to_dict(self) -> dict:
        d: Dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
                             "norm": {"eps": self.norm_eps}, "postln_alpha": self.postln_alpha,
                             "layers": copy.deepcopy(self.layers)}
        if self.max_positions != 1 << 20:
            d["max_positions"] = self.max_positions
        return d

    # --------------------------------------------------------------------- plan
    def _norm_spec(self, name: str) -> PartSpec:
        return PartSpec("rmsnorm", {"size": self.width, "eps": self.norm_eps, "tensor_name": name})

    @staticmethod
    def _rope_spec(rot: dict, dims: int) -> PartSpec:
        return PartSpec("rope", {"theta": float(rot["base"]), "rotary_dim": int(dims), "pairing": "split_half",
                                 "wide_table": True})

    def _mixer_spec(self, i: int) -> PartSpec:
        layer, w = self.layers[i], self.width
        m = layer["mixer"]
        if layer["type"] == "mingru":
            return PartSpec("min_gru", {"hidden_size": w, "inner_size": m["width"]})
        l, r = m["left"], m["right"]
        left = PartSpec("attention", {
            "hidden_size": w, "num_heads": l["heads"], "num_kv_heads": l["kv_heads"], "head_dim": l["dim"],
            "v_head_dim": l["vdim"], "scale": float(l["scale"]), "qkv_bias": True, "o_bias": True,
            "qk_norm": {"eps": self.norm_eps, "over": "row"}, "head_temp": True,
            "position": self._rope_spec(l["rot"], l["rot"]["dims"]), "value_position": self._rope_spec(l["rot"], l["vdim"]),
            "names": {"q": "q", "k": "k", "v": "v", "o": "o", "q_bias": "q.b", "k_bias": "k.b", "v_bias": "v.b",
                      "o_bias": "o.b", "q_norm": "q.norm", "k_norm": "k.norm", "temp": "temp"}})
        right = PartSpec("retention", {
            "hidden_size": w, "num_heads": r["heads"], "key_dim": r["dim"], "value_dim": r["vdim"],
            "decay": [float(v) for v in r["decay"]], "position": self._rope_spec(r["rot"], r["rot"]["dims"]),
            "norm_eps": self.norm_eps})
        return PartSpec("pair", {"hidden_size": w, "left": left, "right": right, "combine": "plain", "joint_projection": True,
                                 "unadded": True, "left_weight": float(m["left_scale"]),
                                 "right_weight": float(m["right_scale"])})

    def _ffn_spec(self, mlp: dict) -> PartSpec:
        return PartSpec("gated_mlp", {"hidden_size": self.width, "intermediate_size": mlp["ff"], "activation": "gelu_tanh",
                                      "bias": True})

    def _layer_spec(self, i: int) -> LayerSpec:
        mlp = self.layers[i].get("mlp")
        parts = {"mixer": SubPart("mixer", self._mixer_spec(i), "mix."), "norm_mixer": SubPart("norm", self._norm_spec("norm1"))}
        if mlp is not None:
            parts["ffn"] = SubPart("ffn", self._ffn_spec(mlp), "mlp.")
            parts["norm_ffn"] = SubPart("norm", self._norm_spec("norm2"))
        return LayerSpec(f"l{i}.", PartSpec("norm_of_sum", {"ffn": mlp is not None, "alpha": self.postln_alpha}), parts)

    def to_plan(self) -> ModelPlan:
        layers = [self._layer_spec(i) for i in range(len(self.layers))]
        plan = ModelPlan(
            architecture=self.architecture, hidden_size=self.width, vocab_size=self.vocab,
            max_positions=self.max_positions,
            embedding=PartSpec("embedding", {"vocab_size": self.vocab, "hidden_size": self.width, "tensor_name": "embed"}),
            layers=layers, schedule=default_schedule(len(layers)), final_norm=self._norm_spec("final.norm"),
            lm_head=PartSpec("lm_head", {"vocab_size": self.vocab, "hidden_size": self.width, "tied": False,
                                         "tensor_name": "head"}),
            final_norm_prefix="", embedding_prefix="", lm_head_prefix="")
        plan.validate()
        return plan
