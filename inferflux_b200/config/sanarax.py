"""Typed configuration of the Sanarax decoder, read from config.json.

Keys: `architecture` ("Sanarax"), `vocab`, `width`, `embedding.scale`, `norm.eps`, `logit_scale` and `layers`, a list whose
entries have `type`, the mixer's sizes under `mixer`, `mlp` (null or {`kind`: `dense`, `ff`}) and optionally `weights_of`
(the layer whose tensors this one runs with; the rest of its entry is that layer's).

    attention         heads, kv_heads, dim, vdim (= dim), scale, rot {base, dims}, mask {size, keep_first}
    latent_attention  heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, rot {base, dims} (dims = rot_dim)
    lightning         heads, dim, vdim, decay (one number a head)

The design, as the plan states it: the embedding's rows are scaled; every sublayer has a norm in front and one behind, with
weights stored as the distance from one; a layer may run several times, every run with a cache and a state of its own.
`attention` is grouped-query attention with biases on queries and keys, values that are the keys in front of the rotation,
halves of a part of every head rotated, a window beside which the sequence's first tokens stay visible, a learned unit in
the softmax's denominator and a gate per head.  `latent_attention` caches a normed latent and one rotated key part that all
heads share; queries go through a normed latent of their own; neighbouring elements rotate; a gate per head.  `lightning`
keeps a matrix of state per head that decays by a constant of the head, with activated queries, keys and values, one norm
over all heads and an elementwise gate.  The feed-forward is two products with a squared ReLU between them.  The model's
norm, a head of its own, scaled logits.  Tensor names: `embed`, `final.norm`, `head`, and per layer i `l<i>.norm1`,
`.norm1b`, `.norm2`, `.norm2b`, `.mix.*`, `.mlp.*`; a bias has its matrix's name with `.b` added.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Dict, List

from .plan import LayerSpec, ModelPlan, PartSpec, ScheduleEntry, SubPart
from .registry import ConfigError, register_architecture

_TYPES = ("attention", "latent_attention", "lightning")
_MLPS = ("dense",)


def _integer(where: str, raw, key: str, least: int = 1) -> int:
    v = raw.get(key) if isinstance(raw, dict) else None
    if isinstance(v, bool) or not isinstance(v, (int, float)) or int(v) != v:
        raise ConfigError(f"config.json (Sanarax): {where}`{key}` must be an integer, got {v!r}")
    if int(v) < least:
        raise ConfigError(f"config.json (Sanarax): {where}`{key}` must be at least {least}, got {v}")
    return int(v)


def _number(where: str, raw, key: str) -> float:
    v = raw.get(key) if isinstance(raw, dict) else None
    if isinstance(v, bool) or not isinstance(v, (int, float)):
        raise ConfigError(f"config.json (Sanarax): {where}`{key}` must be a number, got {v!r}")
    return float(v)


@register_architecture("Sanarax", "sanarax")
@dataclass
class SanaraxConfig:
    vocab: int
    width: int
    layers: List[Dict[str, Any]]
    embedding_scale: float = 1.0
    logit_scale: float = 1.0
    norm_eps: float = 1e-6
    max_positions: int = 1 << 20            # nothing in the design bounds a sequence

    architecture = "Sanarax"
    model_type = "sanarax"

    @property
    def vocab_size(self) -> int:            # the name generic callers use
        return self.vocab

    # ------------------------------------------------------------------ reading
    @classmethod
    def from_dict(cls, raw: dict) -> "SanaraxConfig":
        for key in ("vocab", "width", "layers"):
            if raw.get(key) is None:
                raise ConfigError(f"config.json (Sanarax): missing key `{key}`")
        if not isinstance(raw["layers"], list) or not raw["layers"]:
            raise ConfigError("config.json (Sanarax): `layers` must be a non-empty list")
        emb, norm = raw.get("embedding") or {}, raw.get("norm") or {}
        cfg = cls(
            vocab=_integer("", raw, "vocab"), width=_integer("", raw, "width"), layers=copy.deepcopy(raw["layers"]),
            embedding_scale=_number("embedding.", emb, "scale") if "scale" in emb else 1.0,
            logit_scale=_number("", raw, "logit_scale") if "logit_scale" in raw else 1.0,
            norm_eps=_number("norm.", norm, "eps") if "eps" in norm else 1e-6,
            max_positions=_integer("", raw, "max_positions") if raw.get("max_positions") is not None else 1 << 20)
        cfg.validate()
        return cfg

    def validate(self) -> None:
        if not self.norm_eps > 0:
            raise ConfigError(f"Sanarax config: norm.eps must be positive, got {self.norm_eps}")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]."
            kind = layer.get("type") if isinstance(layer, dict) else None
            if kind not in _TYPES:
                raise ConfigError(f"Sanarax config: {where}type must be one of {_TYPES}, got {kind!r}")
            m = layer.get("mixer")
            if not isinstance(m, dict):
                raise ConfigError(f"Sanarax config: {where}mixer is missing")
            getattr(self, f"_validate_{kind}")(m, where + "mixer.")
            mlp = layer.get("mlp")
            if mlp is not None:
                if not isinstance(mlp, dict) or mlp.get("kind") not in _MLPS:
                    raise ConfigError(f"Sanarax config: {where}mlp.kind must be one of {_MLPS}")
                _integer(where + "mlp.", mlp, "ff")
        for i in range(len(self.layers)):
            self._validate_shared(i)

    def _validate_shared(self, i: int) -> None:
        j = self.layers[i].get("weights_of")
        if j is None:
            return
        where = f"layers[{i}].weights_of"
        if isinstance(j, bool) or not isinstance(j, int) or not 0 <= j < len(self.layers) or j == i:
            raise ConfigError(f"Sanarax config: {where} must name another layer, got {j!r}")
        if self.layers[j].get("weights_of") is not None:
            raise ConfigError(f"Sanarax config: {where} {j} has no tensors of its own")
        for key in ("type", "mixer", "mlp"):
            if self.layers[i].get(key) != self.layers[j].get(key):
                raise ConfigError(f"Sanarax config: {where}: `{key}` is not that of layer {j}")

    @staticmethod
    def _validate_rotation(where: str, m: dict, limit: int) -> None:
        dims = _integer(where + "rot.", m.get("rot"), "dims", least=2)
        if dims % 2 or dims > limit:
            raise ConfigError(f"Sanarax config: {where}rot.dims {dims} must be even and at most {limit}")
        if not _number(where + "rot.", m["rot"], "base") > 0:
            raise ConfigError(f"Sanarax config: {where}rot.base must be positive")

    def _validate_attention(self, m: dict, where: str) -> None:
        for key in ("heads", "kv_heads", "dim"):
            _integer(where, m, key)
        if m["heads"] % m["kv_heads"]:
            raise ConfigError(f"Sanarax config: {where}heads {m['heads']} are not a multiple of kv_heads {m['kv_heads']}")
        if m["dim"] % 2 or m["dim"] > 256:
            raise ConfigError(f"Sanarax config: {where}dim {m['dim']} must be even and at most 256")
        if m.get("vdim") is not None and _integer(where, m, "vdim") != m["dim"]:
            raise ConfigError(f"Sanarax config: {where}vdim {m['vdim']} is not dim {m['dim']} (the values are the keys)")
        if not _number(where, m, "scale") > 0:
            raise ConfigError(f"Sanarax config: {where}scale must be positive")
        self._validate_rotation(where, m, m["dim"])
        if m.get("mask"):
            _integer(where + "mask.", m["mask"], "size")
            if m["mask"].get("keep_first") is not None:
                _integer(where + "mask.", m["mask"], "keep_first", least=0)

    def _validate_latent_attention(self, m: dict, where: str) -> None:
        for key in ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank"):
            _integer(where, m, key)
        if m["kv_rank"] + m["rot_dim"] > 1024:
            raise ConfigError(f"Sanarax config: {where}kv_rank and rot_dim make a cached row longer than the kernels' 1024")
        if not _number(where, m, "scale") > 0:
            raise ConfigError(f"Sanarax config: {where}scale must be positive")
        self._validate_rotation(where, m, m["rot_dim"])

    @staticmethod
    def _validate_lightning(m: dict, where: str) -> None:
        for key in ("heads", "dim", "vdim"):
            _integer(where, m, key)
        if m["dim"] > 512:
            raise ConfigError(f"Sanarax config: {where}dim {m['dim']} is beyond the scan kernel's 512")
        decay = m.get("decay")
        if not isinstance(decay, list) or len(decay) != m["heads"] or not all(
                isinstance(v, (int, float)) and not isinstance(v, bool) for v in decay):
            raise ConfigError(f"Sanarax config: {where}decay must list one number for each of the {m['heads']} heads")

    # ------------------------------------------------------------------ writing
    def to_dict(self) -> dict:
        d: Dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
                             "embedding": {"scale": self.embedding_scale}, "norm": {"eps": self.norm_eps},
                             "logit_scale": self.logit_scale, "layers": copy.deepcopy(self.layers)}
        if self.max_positions != 1 << 20:
            d["max_positions"] = self.max_positions
        return d

    # --------------------------------------------------------------------- plan
    def _norm_spec(self, name: str) -> PartSpec:
        return PartSpec("rmsnorm", {"size": self.width, "eps": self.norm_eps, "unit_offset": True, "tensor_name": name})

    @staticmethod
    def _rope_spec(rot: dict, pairing: str) -> PartSpec:
        return PartSpec("rope", {"theta": float(rot["base"]), "rotary_dim": int(rot["dims"]), "pairing": pairing,
                                 "wide_table": True})

    def _mixer_spec(self, i: int) -> PartSpec:
        layer, w = self.layers[i], self.width
        m = layer["mixer"]
        if layer["type"] == "lightning":
            return PartSpec("lightning", {
                "hidden_size": w, "num_heads": m["heads"], "key_dim": m["dim"], "value_dim": m["vdim"],
                "decay": [float(v) for v in m["decay"]], "norm_eps": self.norm_eps})
        if layer["type"] == "latent_attention":
            return PartSpec("latent_attention", {
                "hidden_size": w, "num_heads": m["heads"], "qk_dim": m["dim"], "rot_dim": m["rot_dim"], "v_dim": m["vdim"],
                "q_rank": m["q_rank"], "kv_rank": m["kv_rank"], "scale": float(m["scale"]), "latent_norm_eps": self.norm_eps,
                "position": self._rope_spec(m["rot"], "interleaved"), "gate": "head"})
        mask = m.get("mask") or {}
        return PartSpec("attention", {
            "hidden_size": w, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"],
            "scale": float(m["scale"]), "qkv_bias": True, "v_from_k": True, "window": mask.get("size"),
            "keep_first": mask.get("keep_first") or 0, "sink": "learned", "gate": "head",
            "position": self._rope_spec(m["rot"], "split_half"),
            "names": {"q": "q", "k": "k", "o": "o", "q_bias": "q.b", "k_bias": "k.b", "sink": "sink", "gate": "g"}})

    def _layer_spec(self, i: int) -> LayerSpec:
        mlp = self.layers[i].get("mlp")
        parts = {"norm_mixer": SubPart("norm", self._norm_spec("norm1")), "mixer": SubPart("mixer", self._mixer_spec(i), "mix."),
                 "postnorm_mixer": SubPart("norm", self._norm_spec("norm1b"))}
        if mlp is not None:
            parts.update({
                "norm_ffn": SubPart("norm", self._norm_spec("norm2")),
                "ffn": SubPart("ffn", PartSpec("up_act_down", {"hidden_size": self.width, "intermediate_size": mlp["ff"],
                                                               "activation": "relu2"}), "mlp."),
                "postnorm_ffn": SubPart("norm", self._norm_spec("norm2b"))})
        return LayerSpec(f"l{i}.", PartSpec("sandwich", {"ffn": mlp is not None, "conv": False}), parts)

    def to_plan(self) -> ModelPlan:
        layers: List[LayerSpec] = []
        made: Dict[int, int] = {}                       # layer with tensors -> its place in the plan
        for i, layer in enumerate(self.layers):
            if layer.get("weights_of") is None:
                made[i] = len(layers)
                layers.append(self._layer_spec(i))
        schedule = [ScheduleEntry(layer=made[i if layer.get("weights_of") is None else layer["weights_of"]], cache=i)
                    for i, layer in enumerate(self.layers)]
        plan = ModelPlan(
            architecture=self.architecture, hidden_size=self.width, vocab_size=self.vocab,
            max_positions=self.max_positions,
            embedding=PartSpec("embedding", {"vocab_size": self.vocab, "hidden_size": self.width, "tensor_name": "embed",
                                             "scale": self.embedding_scale}),
            layers=layers, schedule=schedule, final_norm=self._norm_spec("final.norm"),
            lm_head=PartSpec("lm_head", {"vocab_size": self.vocab, "hidden_size": self.width, "tied": False,
                                         "tensor_name": "head", "scale": self.logit_scale}),
            final_norm_prefix="", embedding_prefix="", lm_head_prefix="")
        plan.validate()
        return plan
