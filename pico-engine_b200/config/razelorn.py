"""Typed configuration of the Razelorn decoder, read from its own config.json keys.

The design: the embedded token times ``embedding.scale``; parallel layers with one layer norm (weight and bias) that both sublayers
read, ``h = norm1(x); x += mixer(h) + ff(h)``.  The mixer is differential attention: every head has two softmax maps over the same
values, with query/key norm per map, rotation of the first ``rot.dims`` entries in the layout of halves with frequencies divided by
wavelength (``rot.scaling``), a sliding window, and the maps' normed difference as the head's output.  The feed-forward is dense,
``down(relu(up h)^2)``; or a mixture of gated silu experts chosen by softmax scores plus a stored correction and weighted by the plain
scores, the last ``router.identity`` of them experts whose output is their input, with a shared expert times a sigmoid; or absent.  A
layer with ``weights_of`` runs another layer's tensors with a cache of its own.  A final layer norm and a head.  Every size and every
constant that may differ between models comes from config.json:

    {"architecture": "Razelorn", "vocab": V, "width": W, "norm": {"eps": e}, "embedding": {"scale": s},
     "layers": [{"type": "attention", "mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "diff", "mask": {"size"},
                 "rot": {"base", "dims", "scaling": {"factor", "low", "high", "original"}}}, "mlp": ..., "weights_of": j}]}
    mlp: null | {"kind": "dense", "ff": F}
       | {"kind": "moe", "router": {"experts", "top", "identity"}, "expert": {"ff"}, "shared": {"ff"}}
"""
from __future__ import annotations

import math
from dataclasses import dataclass, field
from typing import Optional, Tuple

from .registry import register_architecture
from .specs import (ConfigError, DenseMLPSpec, DifferentialAttentionSpec, LayerNormSpec, LayerSpec, MixtureSpec, ModelPlan, NoPositionSpec,
                    RotaryHalvesSpec, ScheduleEntry)

# Positions enter float32 angles: every integer below 2^24 is exact there.
MAX_POSITIONS = 1 << 24


def _int(d, key: str, where: str, least: int = 1) -> int:
    v = d.get(key) if isinstance(d, dict) else None
    if isinstance(v, bool) or not isinstance(v, int) or v < least:
        raise ConfigError(f"{where}{key} must be an integer of at least {least}, found {v!r}")
    return v


def _number(d, key: str, where: str, positive: bool = True) -> float:
    v = d.get(key) if isinstance(d, dict) else None
    if isinstance(v, bool) or not isinstance(v, (int, float)) or not math.isfinite(v) or (positive and not v > 0):
        raise ConfigError(f"{where}{key} must be a {'positive ' if positive else ''}number, found {v!r}")
    return float(v)


def _rot(m: dict, where: str) -> Optional[dict]:
    rot = m.get("rot")
    if rot is None:
        return None
    out = {"base": _number(rot, "base", where + "rot."), "dims": _int(rot, "dims", where + "rot.", least=0)}
    if out["dims"] % 2 or out["dims"] > m["dim"]:
        raise ConfigError(f"{where}rot.dims must be even and at most dim = {m['dim']}, found {out['dims']}")
    sc = rot.get("scaling")
    if sc is not None:
        out["scaling"] = {k: _number(sc, k, where + "rot.scaling.") for k in ("factor", "high", "low", "original")}
        if not out["scaling"]["low"] < out["scaling"]["high"]:
            raise ConfigError(f"{where}rot.scaling.low must lie below high, found {out['scaling']['low']} and {out['scaling']['high']}")
    return out


def _attention(m: dict, where: str) -> dict:
    out = {k: _int(m, k, where) for k in ("heads", "kv_heads", "dim", "vdim")}
    out["scale"] = _number(m, "scale", where)
    out["diff"] = _number(m, "diff", where, positive=False)
    if out["heads"] % out["kv_heads"]:
        raise ConfigError(f"{where}: {out['heads']} heads cannot share {out['kv_heads']} key/value heads evenly")
    rot = _rot(m, where)
    if rot is not None:
        out["rot"] = rot
    if m.get("mask") is not None:
        out["mask"] = {"size": _int(m["mask"], "size", where + "mask.")}
    return out


def _mlp(mlp, where: str) -> Optional[dict]:
    if mlp is None:
        return None
    if not isinstance(mlp, dict) or mlp.get("kind") not in ("dense", "moe"):
        raise ConfigError(f"{where}kind must be \"dense\" or \"moe\" (or mlp null), found {mlp!r}")
    if mlp["kind"] == "dense":
        return {"ff": _int(mlp, "ff", where), "kind": "dense"}
    router = mlp.get("router")
    r = {"experts": _int(router, "experts", where + "router."), "top": _int(router, "top", where + "router.")}
    if router.get("identity") is not None:
        r["identity"] = _int(router, "identity", where + "router.", least=0)
    if r["top"] > r["experts"] + r.get("identity", 0):
        raise ConfigError(f"{where}router.top = {r['top']} exceeds the router's {r['experts'] + r.get('identity', 0)} outputs")
    out = {"expert": {"ff": _int(mlp.get("expert"), "ff", where + "expert.")}, "kind": "moe", "router": r}
    if mlp.get("shared") is not None:
        out["shared"] = {"ff": _int(mlp["shared"], "ff", where + "shared.")}
    return out


@dataclass(frozen=True)
class RazelornLayer:
    """One entry of ``layers``: the checked ``mixer`` and ``mlp`` objects as config.json spells them, and the layer whose tensors it uses."""
    mixer: dict = field(hash=False)
    mlp: Optional[dict] = field(default=None, hash=False)
    weights_of: Optional[int] = None

    @classmethod
    def from_dict(cls, d: dict, i: int) -> "RazelornLayer":
        where = f"layers[{i}]."
        if not isinstance(d, dict) or d.get("type") != "attention":
            raise ConfigError(f"{where}type must be \"attention\", found {d.get('type') if isinstance(d, dict) else d!r}")
        if not isinstance(d.get("mixer"), dict):
            raise ConfigError(f"{where}mixer must be an object with the mixer's sizes")
        of = None if d.get("weights_of") is None else _int(d, "weights_of", where, least=0)
        return cls(_attention(d["mixer"], where + "mixer."), _mlp(d.get("mlp"), where + "mlp."), of)

    def to_dict(self) -> dict:
        d = {"mixer": dict(self.mixer), "mlp": self.mlp, "type": "attention"}
        if self.weights_of is not None:
            d["weights_of"] = self.weights_of
        return d


@dataclass(frozen=True)
class RazelornConfig:
    ARCHITECTURE = "Razelorn"

    vocab: int
    width: int
    layers: Tuple[RazelornLayer, ...]
    norm_eps: float
    embedding_scale: float = 1.0

    @classmethod
    def from_dict(cls, d: dict) -> "RazelornConfig":
        missing = [k for k in ("vocab", "width", "layers", "norm") if d.get(k) is None]
        if missing:
            raise ConfigError("config.json lacks " + ", ".join(missing))
        if not isinstance(d["layers"], list) or not d["layers"]:
            raise ConfigError("layers must be a non-empty list")
        if not isinstance(d["norm"], dict):
            raise ConfigError("norm must be an object ({\"eps\": ...})")
        emb = d.get("embedding")
        scale = 1.0 if not isinstance(emb, dict) or emb.get("scale") is None else _number(emb, "scale", "embedding.")
        cfg = cls(vocab=_int(d, "vocab", ""), width=_int(d, "width", ""),
                  layers=tuple(RazelornLayer.from_dict(x, i) for i, x in enumerate(d["layers"])),
                  norm_eps=_number(d["norm"], "eps", "norm."), embedding_scale=scale)
        for i, x in enumerate(cfg.layers):
            j = cfg.owner(i)
            if (cfg.layers[j].mixer, cfg.layers[j].mlp) != (x.mixer, x.mlp):
                raise ConfigError(f"layers[{i}] uses the tensors of layer {j} (weights_of), but its mixer or mlp is another")
        return cfg

    def owner(self, i: int) -> int:
        """The layer whose tensors layer ``i`` uses (itself, or the end of the chain of ``weights_of``)."""
        seen = {i}
        while self.layers[i].weights_of is not None:
            j = self.layers[i].weights_of
            if j >= len(self.layers) or j in seen:
                raise ConfigError(f"layers[{i}].weights_of = {j} names no layer with tensors of its own")
            seen.add(j)
            i = j
        return i

    def to_dict(self) -> dict:
        return {"architecture": self.ARCHITECTURE, "embedding": {"scale": self.embedding_scale},
                "layers": [x.to_dict() for x in self.layers], "norm": {"eps": self.norm_eps}, "vocab": self.vocab, "width": self.width}

    # ---------------------------------------------------------------- the plan

    def _mixer_spec(self, m: dict, p: str) -> DifferentialAttentionSpec:
        rot, position = m.get("rot"), NoPositionSpec()
        if rot is not None and rot["dims"]:
            sc = rot.get("scaling")
            position = RotaryHalvesSpec(head_dim=m["dim"], dims=rot["dims"], base=rot["base"],
                                        bands=None if sc is None else (sc["factor"], sc["low"], sc["high"], sc["original"]))
        return DifferentialAttentionSpec(hidden=self.width, n_heads=m["heads"], n_kv_heads=m["kv_heads"], head_dim=m["dim"],
                                         v_head_dim=m["vdim"], window=(m.get("mask") or {}).get("size"), scale=m["scale"], position=position,
                                         prefix=p, lambda_base=m["diff"], out_scale=1.0 - m["diff"], norm_eps=self.norm_eps)

    def _ff_spec(self, mlp: Optional[dict], p: str):
        if mlp is None:
            return None
        if mlp["kind"] == "dense":
            return DenseMLPSpec(self.width, mlp["ff"], p, activation="relu2")
        r = mlp["router"]
        return MixtureSpec(hidden=self.width, n_experts=r["experts"], top_k=r["top"], intermediate=mlp["expert"]["ff"], prefix=p,
                           activation="silu", shared_intermediate=(mlp.get("shared") or {}).get("ff"), scores="softmax_all",
                           correction_name="correction", n_identity=r.get("identity", 0))

    def plan(self) -> ModelPlan:
        W, eps = self.width, self.norm_eps
        layers, at = [], {}
        for i, x in enumerate(self.layers):
            if self.owner(i) == i:
                p = f"l{i}."
                at[i] = len(layers)
                layers.append(LayerSpec(mixer=self._mixer_spec(x.mixer, p + "mix."), mixer_norm=LayerNormSpec(W, eps, p + "norm1", p + "norm1.b"),
                                        feed_forward=self._ff_spec(x.mlp, p + "mlp."), arrangement="parallel_one_norm"))
        plan = ModelPlan(architecture=self.ARCHITECTURE, vocab_size=self.vocab, hidden_size=W, embedding="embed", layers=tuple(layers),
                         schedule=tuple(ScheduleEntry(at[self.owner(i)]) for i in range(len(self.layers))),
                         final_norm=LayerNormSpec(W, eps, "final.norm", "final.norm.b"), head="head", max_positions=MAX_POSITIONS,
                         embedding_scale=self.embedding_scale)
        plan.validate()
        return plan


register_architecture(RazelornConfig.ARCHITECTURE, RazelornConfig)
