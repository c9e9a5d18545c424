"""Typed configuration of the Bibalix architecture: a pre-norm decoder (layer norms with weight and
bias, the head tied to the embedding) with two kinds of mixer.  `attention`: attention in two maps
(two queries and two keys per head over the same values, projections with biases, an RMS norm per
query and key, rotated halves, a sliding window beside which the first tokens stay visible, the
second map's output times a learned number taken off the first's, an RMS norm per head without a
weight, a sigmoid gate per head).  `latent_attention`: queries straight from the input, a cached
key/value latent with a rotated key part shared by the heads (halves, ramped frequency scaling), a
sliding window, a sigmoid gate per head.  Feed-forwards are dense gated ones (gelu's tanh form) or
mixtures of clamped gated experts under a softmax router whose scores, times a constant, are the
weights, beside a shared expert behind a gate per token; either may be absent.

config.json gives `architecture`, `vocab`, `width`, `norm.eps` and `layers`: per layer `type`
("attention" or "latent_attention"), `mixer` (its sizes) and `mlp` (null, {"kind": "dense", ff} or
{"kind": "moe", "expert": {ff, limit}, "router": {experts, top, scale}, "shared": {ff, limit} | absent}).
attention: heads, kv_heads, dim (of one map), vdim, scale, diff, mask: {size, keep_first} | absent, rot:
{dims, base}.  latent_attention: heads, dim, rot_dim, vdim, kv_rank, scale, mask: {size} | absent,
rot: {dims = rot_dim, base, scaling: {factor, original, fast, slow} | absent}.

Tensor names (`.b`: the bias of the same name): `embed`, `final.norm` `.b`; per layer `l<i>.`: `norm1` `.b`,
`norm2` `.b` (with a feed-forward); attention `mix.{q, k, v}` `.b`, `mix.{q.norm, k.norm, lq1, lk1, lq2, lk2,
g, o}`; latent_attention `mix.{q, dkv, dkv.norm, uk, uv, g, o}`; dense `mlp.{gate, up, down}`; moe
`mlp.router`, `mlp.e<j>.{gate, up, down}`, `mlp.shared.{gate, up, down, sg}`.
"""

from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Any

from .qwen2 import ConfigError
from .spec import LayerSpec, ModelSpec, PartSpec, RunSpec

ARCHITECTURE = "Bibalix"
DEFAULT_MAX_POSITIONS = 1 << 20   # positions are computed, not learned: a bound for tables only
MIXER_TYPES = ("attention", "latent_attention")
EXPERT_SLOPE = 1.702              # the experts' g * sigmoid(1.702 g) * (u + 1)
EXPERT_SHIFT = 1.0
SCALING_KEYS = ("factor", "original", "fast", "slow")


def _int(d: Any, key: str, where: str, least: int = 1) -> int:
    v = d.get(key) if isinstance(d, dict) else None
    if not isinstance(v, int) or isinstance(v, bool) or v < least:
        raise ConfigError(f"config.json: {where}{key} must be an integer >= {least}, got {v!r}")
    return v


def _number(d: Any, key: str, where: str) -> float:
    v = d.get(key) if isinstance(d, dict) else None
    if not isinstance(v, (int, float)) or isinstance(v, bool):
        raise ConfigError(f"config.json: {where}{key} must be a number, got {v!r}")
    return float(v)


def _positive(d: Any, key: str, where: str) -> float:
    v = _number(d, key, where)
    if not v > 0.0:
        raise ConfigError(f"config.json: {where}{key} must be positive")
    return v


def _rotation(m: dict, where: str, width: int) -> dict[str, Any]:
    w = where + "rot."
    rot = m.get("rot")
    out: dict[str, Any] = {"dims": _int(rot, "dims", w, 0), "base": _positive(rot, "base", w)}
    if out["dims"] % 2 or out["dims"] > width:
        raise ConfigError(f"config.json: {w}dims must be even and at most {width}")
    if rot.get("scaling") is not None:
        out["scaling"] = {k: _positive(rot["scaling"], k, w + "scaling.") for k in SCALING_KEYS}
    return out


def _rotary(rot: dict[str, Any]) -> dict[str, Any]:
    out = {"dims": rot["dims"], "base": rot["base"]}
    if rot.get("scaling") is not None:
        out["scaling"] = {"kind": "ramp", **rot["scaling"]}
    return out


@dataclass(frozen=True)
class BibalixLayerConfig:
    type: str                    # one of MIXER_TYPES
    mixer: dict[str, Any]        # the mixer's sizes, as the file gives them (validated)
    mlp: dict[str, Any] | None   # None: the layer has no feed-forward


@dataclass(frozen=True)
class BibalixConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: tuple[BibalixLayerConfig, ...]
    max_positions: int = DEFAULT_MAX_POSITIONS
    eos_token_id: int | None = None

    architecture = ARCHITECTURE

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    # ---------------------------------------------------------------- reading
    @staticmethod
    def _mixer(kind: str, m: Any, where: str) -> dict[str, Any]:
        if not isinstance(m, dict):
            raise ConfigError(f"config.json: {where}mixer must be an object")
        w = where + "mixer."
        mask = m.get("mask")
        if kind == "attention":
            out: dict[str, Any] = {k: _int(m, k, w) for k in ("heads", "kv_heads", "dim", "vdim")}
            out["scale"], out["diff"] = _number(m, "scale", w), _number(m, "diff", w)
            if out["heads"] % out["kv_heads"]:
                raise ConfigError(f"config.json: {w}heads must be a multiple of kv_heads")
            if mask is not None:
                out["mask"] = {"size": _int(mask, "size", w + "mask.")}
                if mask.get("keep_first") is not None:
                    out["mask"]["keep_first"] = _int(mask, "keep_first", w + "mask.", 0)
            out["rot"] = _rotation(m, w, out["dim"])
            return out
        out = {k: _int(m, k, w) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank")}
        out["scale"] = _number(m, "scale", w)
        if mask is not None:
            out["mask"] = {"size": _int(mask, "size", w + "mask.")}
        out["rot"] = _rotation(m, w, out["rot_dim"])
        if out["rot"]["dims"] != out["rot_dim"]:
            raise ConfigError(f"config.json: {w}rot.dims must be rot_dim")
        return out

    @staticmethod
    def _mlp(mlp: Any, where: str) -> dict[str, Any] | None:
        if mlp is None:
            return None
        w = where + "mlp."
        kind = mlp.get("kind") if isinstance(mlp, dict) else None
        if kind == "dense":
            return {"kind": "dense", "ff": _int(mlp, "ff", w)}
        if kind != "moe":
            raise ConfigError(f"config.json: {where}mlp must be null or of kind 'dense' or 'moe'")

        def expert(key: str) -> dict[str, Any]:
            return {"ff": _int(mlp.get(key), "ff", f"{w}{key}."), "limit": _positive(mlp.get(key), "limit", f"{w}{key}.")}
        r = mlp.get("router")
        router: dict[str, Any] = {"experts": _int(r, "experts", w + "router."),
                                  "top": _int(r, "top", w + "router.")}
        if router["top"] > router["experts"]:
            raise ConfigError(f"config.json: {w}router.top exceeds the number of experts")
        if r.get("scale") is not None:
            router["scale"] = _number(r, "scale", w + "router.")
        out = {"kind": "moe", "expert": expert("expert"), "router": router}
        if mlp.get("shared") is not None:
            out["shared"] = expert("shared")
        return out

    @classmethod
    def from_dict(cls, d: dict[str, Any]) -> "BibalixConfig":
        missing = [k for k in ("vocab", "width", "norm", "layers") if k not in d]
        if missing:
            raise ConfigError("config.json lacks: " + ", ".join(missing))
        if not isinstance(d["layers"], list) or not d["layers"]:
            raise ConfigError("config.json: layers must be a non-empty list")
        layers = []
        for i, raw in enumerate(d["layers"]):
            where = f"layers[{i}]."
            if not isinstance(raw, dict) or "type" not in raw or "mixer" not in raw:
                raise ConfigError(f"config.json: {where[:-1]} needs 'type' and 'mixer'")
            if raw["type"] not in MIXER_TYPES:
                raise ConfigError(f"config.json: {where}type {raw['type']!r} is not a mixer of this "
                                  f"architecture (known: {', '.join(MIXER_TYPES)})")
            layers.append(BibalixLayerConfig(raw["type"], cls._mixer(raw["type"], raw["mixer"], where),
                                             cls._mlp(raw.get("mlp"), where)))
        cfg = cls(vocab=_int(d, "vocab", ""), width=_int(d, "width", ""),
                  norm_eps=_number(d["norm"], "eps", "norm."), layers=tuple(layers),
                  max_positions=int(d.get("max_positions", DEFAULT_MAX_POSITIONS)),
                  eos_token_id=d.get("eos_token_id"))
        cfg.validate()
        return cfg

    @classmethod
    def from_json(cls, path: str) -> "BibalixConfig":
        if os.path.isdir(path):
            path = os.path.join(path, "config.json")
        with open(path, "r", encoding="utf-8") as f:
            return cls.from_dict(json.load(f))

    def to_dict(self) -> dict[str, Any]:
        d: dict[str, Any] = {
            "architecture": ARCHITECTURE, "vocab": self.vocab, "width": self.width,
            "norm": {"eps": self.norm_eps},
            "layers": [{"type": l.type, "mixer": json.loads(json.dumps(l.mixer)),
                        "mlp": None if l.mlp is None else json.loads(json.dumps(l.mlp))}
                       for l in self.layers]}
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            d["max_positions"] = self.max_positions
        if self.eos_token_id is not None:
            d["eos_token_id"] = self.eos_token_id
        return d

    # ------------------------------------------------------------- validation
    def validate(self) -> None:
        if not self.norm_eps > 0.0:
            raise ConfigError("norm.eps must be positive")
        if self.max_positions <= 0:
            raise ConfigError("max_positions must be positive")

    # ------------------------------------------------------------ model spec
    def _mixer_spec(self, p: str, layer: BibalixLayerConfig) -> PartSpec:
        D, eps, m = self.width, self.norm_eps, layer.mixer
        mask = m.get("mask")
        if layer.type == "attention":
            names = {"q_norm": f"{p}.mix.q.norm", "k_norm": f"{p}.mix.k.norm", "gate_weight": f"{p}.mix.g",
                     "o_weight": f"{p}.mix.o"}
            for part in ("q", "k", "v"):
                names.update({f"{part}_weight": f"{p}.mix.{part}", f"{part}_bias": f"{p}.mix.{part}.b"})
            for part in ("lq1", "lk1", "lq2", "lk2"):
                names[part] = f"{p}.mix.{part}"
            return PartSpec("differential_attention", {
                "hidden_size": D, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"],
                "key_dim": m["dim"], "value_dim": m["vdim"], "scale": m["scale"], "start": m["diff"],
                "qkv_bias": True, "head_norm": True, "head_gate": True, "eps": eps,
                "rotary": _rotary(m["rot"]),
                "mask": None if mask is None else {"kind": "window", "size": mask["size"],
                                                   "keep_first": mask.get("keep_first", 0)},
                "names": names})
        return PartSpec("latent_attention", {
            "hidden_size": D, "heads": m["heads"], "key_dim": m["dim"], "value_dim": m["vdim"],
            "q_rank": None, "kv_rank": m["kv_rank"], "rot_dim": m["rot_dim"], "rotary": _rotary(m["rot"]),
            "scale": m["scale"], "eps": eps, "window": None if mask is None else mask["size"],
            "sink": False, "own_latent": True, "gate": "head",
            "names": {"q": f"{p}.mix.q", "kv_down": f"{p}.mix.dkv", "kv_norm": f"{p}.mix.dkv.norm",
                      "k_up": f"{p}.mix.uk", "v_up": f"{p}.mix.uv", "gate": f"{p}.mix.g",
                      "out": f"{p}.mix.o"}})

    def _ff_spec(self, p: str, mlp: dict[str, Any]) -> PartSpec:
        D = self.width
        if mlp["kind"] == "dense":
            return PartSpec("clamped_glu", {
                "hidden_size": D, "intermediate_size": mlp["ff"], "activation": "gelu_tanh",
                "names": {"gate_weight": f"{p}.mlp.gate", "up_weight": f"{p}.mlp.up",
                          "down_weight": f"{p}.mlp.down"}})

        def form(e: dict[str, Any]) -> dict[str, float]:
            return {"limit": e["limit"], "alpha": EXPERT_SLOPE, "shift": EXPERT_SHIFT}
        r, experts = mlp["router"], range(mlp["router"]["experts"])
        names: dict[str, Any] = {"router": f"{p}.mlp.router",
                                 "gate": [f"{p}.mlp.e{e}.gate" for e in experts],
                                 "up": [f"{p}.mlp.e{e}.up" for e in experts],
                                 "down": [f"{p}.mlp.e{e}.down" for e in experts]}
        shared = mlp.get("shared")
        if shared is not None:
            names.update({"shared_gate": f"{p}.mlp.shared.gate", "shared_up": f"{p}.mlp.shared.up",
                          "shared_down": f"{p}.mlp.shared.down", "shared_token_gate": f"{p}.mlp.shared.sg"})
        return PartSpec("routed_moe", {
            "hidden_size": D, "experts": r["experts"], "top": r["top"], "factor": r.get("scale", 1.0),
            "expert_ff": mlp["expert"]["ff"], "gated": form(mlp["expert"]),
            "shared": None if shared is None else {"ff": shared["ff"], "gated": form(shared), "token_gate": True},
            "names": names})

    def to_model_spec(self) -> ModelSpec:
        D = self.width

        def norm(name: str) -> PartSpec:
            return PartSpec("layernorm", {"size": D, "eps": self.norm_eps,
                                          "names": {"weight": name, "bias": f"{name}.b"}})

        layers = []
        for i, layer in enumerate(self.layers):
            p = f"l{i}"
            norms = {"mixer": norm(f"{p}.norm1")}
            ff = None
            if layer.mlp is not None:
                ff = self._ff_spec(p, layer.mlp)
                norms["feed_forward"] = norm(f"{p}.norm2")
            layers.append(LayerSpec(prefix=p, mixer=self._mixer_spec(p, layer), feed_forward=ff,
                                    norms=norms, arrangement="pre_norm"))
        spec = ModelSpec(
            architecture=ARCHITECTURE, hidden_size=D, vocab_size=self.vocab,
            max_positions=self.max_positions,
            embedding=PartSpec("token_embedding", {"vocab_size": self.vocab, "hidden_size": D,
                                                   "scale": 1.0, "names": {"weight": "embed"}}),
            layers=tuple(layers), schedule=tuple(RunSpec(i) for i in range(len(self.layers))),
            final_norm=norm("final.norm"),
            head=PartSpec("lm_head", {"vocab_size": self.vocab, "hidden_size": D, "tied": True,
                                      "names": {"weight": "head", "tied_to": "embed"}}))
        spec.validate()
        return spec
