"""Typed configuration of the Dosuvik architecture: a decoder whose sublayers read the residual
stream itself and are normed on their way back, x <- x + norm(sublayer(x)) (RMS norms whose weight is
stored as what the factor exceeds one by), and whose stream is replaced behind every layer by a
learned weighted sum of the embedding's output and all layers' results so far.  Three kinds of
mixer: sliding-window attention (an RMS norm over all query rows and one over all key rows, rotated
halves, values that are turned by position and turned back behind the softmax, a learned sink per
head); latent attention (queries straight from the input, a cached key/value latent with a rotated
key part shared by the heads, a sigmoid gate per output element); and retention (rotated queries and
keys, a float32 matrix per head with a constant decay, an RMS norm per head without a weight, a
SiLU gate).  Feed-forwards are dense with a clamped gated activation, or mixtures of experts
whose router takes sigmoid scores, a correction for the choice only, and groups of experts ranked by
their two best members; either may be absent.

config.json gives `architecture`, `vocab`, `width`, `norm.eps` and `layers`: per layer `type`
("attention", "latent_attention" or "retention"), `mixer` (its sizes) and `mlp` (null, {"kind": "dense",
ff, limit} or {"kind": "moe", "expert": {ff}, "router": {experts, top, groups: {count, keep} |
absent}}).  attention: heads, kv_heads, dim, vdim, scale, mask: {size} | absent, rot: {dims, base}.
latent_attention: heads, dim, rot_dim, vdim, kv_rank, scale, rot: {dims = rot_dim, base}.  retention:
heads, dim, vdim, decay (one number per head), rot: {dims, base}.

Tensor names: `embed`, `final.norm`, `head`; per layer `l<i>.`: `norm1`, `norm2` (with a feed-forward),
`dwa` [i + 2]; attention `mix.{q, k, v, q.norm, k.norm, sink, o}`; latent_attention `mix.{q, dkv, dkv.norm,
uk, uv, g, o}`; retention `mix.{q, k, v, g, o}`; dense `mlp.{gate, up, down}`; moe `mlp.{router, correction}`,
`mlp.e<j>.{gate, up, down}`.
"""

from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Any

from .qwen2 import ConfigError
from .spec import LayerSpec, ModelSpec, PartSpec, RunSpec

ARCHITECTURE = "Dosuvik"
DEFAULT_MAX_POSITIONS = 1 << 20   # positions are computed, not learned: a bound for tables only
MIXER_TYPES = ("attention", "latent_attention", "retention")
ACTIVATION_SLOPE = 1.702          # the dense feed-forward's g * sigmoid(1.702 g) * (u + 1)
ACTIVATION_SHIFT = 1.0


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


def _rotation(m: dict, where: str, width: int) -> dict[str, Any]:
    w = where + "rot."
    rot = m.get("rot")
    out = {"dims": _int(rot, "dims", w, 0), "base": _number(rot, "base", w)}
    if out["dims"] % 2 or out["dims"] > width:
        raise ConfigError(f"config.json: {w}dims must be even and at most {width}")
    if not out["base"] > 0.0:
        raise ConfigError(f"config.json: {w}base must be positive")
    return out


@dataclass(frozen=True)
class DosuvikLayerConfig:
    type: str                    # one of MIXER_TYPES
    mixer: dict[str, Any]        # the mixer's sizes, as the file gives them (validated)
    mlp: dict[str, Any] | None   # None: the layer has no feed-forward


@dataclass(frozen=True)
class DosuvikConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: tuple[DosuvikLayerConfig, ...]
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
        if kind == "attention":
            out: dict[str, Any] = {k: _int(m, k, w) for k in ("heads", "kv_heads", "dim", "vdim")}
            out["scale"] = _number(m, "scale", w)
            if out["heads"] % out["kv_heads"]:
                raise ConfigError(f"config.json: {w}heads must be a multiple of kv_heads")
            if out["vdim"] % 2:
                raise ConfigError(f"config.json: {w}vdim must be even: values are turned in pairs")
            if m.get("mask") is not None:
                out["mask"] = {"size": _int(m["mask"], "size", w + "mask.")}
            out["rot"] = _rotation(m, w, out["dim"])
            return out
        if kind == "latent_attention":
            out = {k: _int(m, k, w) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank")}
            out["scale"] = _number(m, "scale", w)
            out["rot"] = _rotation(m, w, out["rot_dim"])
            if out["rot"]["dims"] != out["rot_dim"]:
                raise ConfigError(f"config.json: {w}rot.dims must be rot_dim")
            return out
        out = {k: _int(m, k, w) for k in ("heads", "dim", "vdim")}
        decay = m.get("decay")
        if not isinstance(decay, list) or len(decay) != out["heads"]:
            raise ConfigError(f"config.json: {w}decay must list one number per head")
        out["decay"] = [_number({"decay": v}, "decay", w) for v in decay]
        out["rot"] = _rotation(m, w, out["dim"])
        return out

    @staticmethod
    def _mlp(mlp: Any, where: str) -> dict[str, Any] | None:
        if mlp is None:
            return None
        w = where + "mlp."
        kind = mlp.get("kind") if isinstance(mlp, dict) else None
        if kind == "dense":
            out = {"kind": "dense", "ff": _int(mlp, "ff", w), "limit": _number(mlp, "limit", w)}
            if not out["limit"] > 0.0:
                raise ConfigError(f"config.json: {w}limit must be positive")
            return out
        if kind != "moe":
            raise ConfigError(f"config.json: {where}mlp must be null or of kind 'dense' or 'moe'")
        r = mlp.get("router")
        router: dict[str, Any] = {"experts": _int(r, "experts", w + "router."),
                                  "top": _int(r, "top", w + "router.")}
        reachable = router["experts"]
        if r.get("groups") is not None:
            g = w + "router.groups."
            groups = {"count": _int(r["groups"], "count", g), "keep": _int(r["groups"], "keep", g)}
            if router["experts"] % groups["count"] or groups["keep"] > groups["count"]:
                raise ConfigError(f"config.json: {g}count must divide experts and keep must not exceed it")
            router["groups"] = groups
            reachable = groups["keep"] * (router["experts"] // groups["count"])
        if router["top"] > reachable:
            raise ConfigError(f"config.json: {w}router.top exceeds the experts that can be chosen")
        return {"kind": "moe", "expert": {"ff": _int(mlp.get("expert"), "ff", w + "expert.")},
                "router": router}

    @classmethod
    def from_dict(cls, d: dict[str, Any]) -> "DosuvikConfig":
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
            layers.append(DosuvikLayerConfig(raw["type"], cls._mixer(raw["type"], raw["mixer"], where),
                                             cls._mlp(raw.get("mlp"), where)))
        cfg = cls(vocab=_int(d, "vocab", ""), width=_int(d, "width", ""),
                  norm_eps=_number(d["norm"], "eps", "norm."), layers=tuple(layers),
                  max_positions=int(d.get("max_positions", DEFAULT_MAX_POSITIONS)),
                  eos_token_id=d.get("eos_token_id"))
        cfg.validate()
        return cfg

    @classmethod
    def from_json(cls, path: str) -> "DosuvikConfig":
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
    def _mixer_spec(self, p: str, layer: DosuvikLayerConfig) -> PartSpec:
        D, eps, m = self.width, self.norm_eps, layer.mixer
        names = {"q_weight": f"{p}.mix.q", "k_weight": f"{p}.mix.k", "v_weight": f"{p}.mix.v",
                 "o_weight": f"{p}.mix.o"}
        if layer.type == "attention":
            mask = m.get("mask")
            return PartSpec("normed_attention", {
                "hidden_size": D, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"],
                "key_dim": m["dim"], "value_dim": m["vdim"], "scale": m["scale"], "qkv_bias": False,
                "row_norm": True, "eps": eps, "rotary": dict(m["rot"]), "turn_values": True,
                "mask": None if mask is None else {"kind": "window", "size": mask["size"]},
                "sink": "learned",
                "names": {**names, "q_norm": f"{p}.mix.q.norm", "k_norm": f"{p}.mix.k.norm",
                          "sink": f"{p}.mix.sink"}})
        if layer.type == "latent_attention":
            return PartSpec("latent_attention", {
                "hidden_size": D, "heads": m["heads"], "key_dim": m["dim"], "value_dim": m["vdim"],
                "q_rank": None, "kv_rank": m["kv_rank"], "rot_dim": m["rot_dim"],
                "rotary": {**m["rot"], "neighbours": True}, "scale": m["scale"], "eps": eps,
                "window": None, "sink": False, "own_latent": True, "gate": True,
                "names": {"q": f"{p}.mix.q", "kv_down": f"{p}.mix.dkv", "kv_norm": f"{p}.mix.dkv.norm",
                          "k_up": f"{p}.mix.uk", "v_up": f"{p}.mix.uv", "gate": f"{p}.mix.g",
                          "out": f"{p}.mix.o"}})
        return PartSpec("retention", {
            "hidden_size": D, "heads": m["heads"], "key_dim": m["dim"], "value_dim": m["vdim"],
            "decay": list(m["decay"]), "rotary": dict(m["rot"]), "k_scale": m["dim"] ** -0.5, "eps": eps,
            "names": {**names, "gate_weight": f"{p}.mix.g"}})

    def _ff_spec(self, p: str, mlp: dict[str, Any]) -> PartSpec:
        D = self.width
        if mlp["kind"] == "dense":
            return PartSpec("clamped_glu", {
                "hidden_size": D, "intermediate_size": mlp["ff"], "limit": mlp["limit"],
                "alpha": ACTIVATION_SLOPE, "shift": ACTIVATION_SHIFT,
                "names": {"gate_weight": f"{p}.mlp.gate", "up_weight": f"{p}.mlp.up",
                          "down_weight": f"{p}.mlp.down"}})
        r, experts = mlp["router"], range(mlp["router"]["experts"])
        groups = None if r.get("groups") is None else {**r["groups"], "best": 2}
        return PartSpec("routed_moe", {
            "hidden_size": D, "experts": r["experts"], "top": r["top"], "expert_ff": mlp["expert"]["ff"],
            "scores": "sigmoid", "correction": True, "groups": groups,
            "names": {"router": f"{p}.mlp.router", "correction": f"{p}.mlp.correction",
                      "gate": [f"{p}.mlp.e{e}.gate" for e in experts],
                      "up": [f"{p}.mlp.e{e}.up" for e in experts],
                      "down": [f"{p}.mlp.e{e}.down" for e in experts]}})

    def to_model_spec(self) -> ModelSpec:
        D = self.width

        def norm(name: str) -> PartSpec:
            return PartSpec("rmsnorm", {"size": D, "eps": self.norm_eps, "offset": 1.0,
                                        "names": {"weight": name}})

        plain = PartSpec("none", {"size": D})
        layers = []
        for i, layer in enumerate(self.layers):
            p = f"l{i}"
            norms = {"mixer": plain, "mixer_post": norm(f"{p}.norm1")}
            ff = None
            if layer.mlp is not None:
                ff = self._ff_spec(p, layer.mlp)
                norms.update({"feed_forward": plain, "feed_forward_post": norm(f"{p}.norm2")})
            layers.append(LayerSpec(prefix=p, mixer=self._mixer_spec(p, layer), feed_forward=ff,
                                    norms=norms, arrangement="sandwich_norm"))
        n = len(self.layers)
        spec = ModelSpec(
            architecture=ARCHITECTURE, hidden_size=D, vocab_size=self.vocab,
            max_positions=self.max_positions,
            embedding=PartSpec("token_embedding", {"vocab_size": self.vocab, "hidden_size": D,
                                                   "scale": 1.0, "names": {"weight": "embed"}}),
            layers=tuple(layers),
            schedule=tuple(RunSpec(i, average=f"depth{i}") for i in range(n)),
            final_norm=norm("final.norm"),
            head=PartSpec("lm_head", {"vocab_size": self.vocab, "hidden_size": D, "tied": False,
                                      "names": {"weight": "head", "tied_to": "embed"}}),
            stream_parts={f"depth{i}": PartSpec("depth_average", {"count": i + 2,
                                                                  "names": {"weight": f"l{i}.dwa"}})
                          for i in range(n)})
        spec.validate()
        return spec
