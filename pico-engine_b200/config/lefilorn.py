"""Typed configuration of the Lefilorn decoder, read from its own config.json keys.

The design: the embedded token times ``embedding.scale``; a residual of ``streams`` streams, all equal to that at first.  A sublayer
reads the RMS-normed weighted sum of the streams, and its output and the old streams make the new ones (``l<i>.hc1.*`` around the
mixer, ``l<i>.hc2.*`` around the feed-forward); what leaves the last layer is the sum of the streams.  Every layer's mixer is
``"parallel"``: two mixers on the same input, left_scale * left + right_scale * right.  Left: grouped softmax attention with biases on
q, k and v, an RMS norm over all query rows and one over all key rows before the rotation of neighbours, a sliding window that keeps a
sequence's first keys visible, and a sigmoid gate on the concatenated heads.  Right: linear attention with a fixed decay per head and
rotation of halves, keys times dim^(-1/2), every head's output divided by its root mean square, a silu gate.  The feed-forward is
``down(relu(gate h) * (up h))``, or absent.  A run of layers may be repeated with the same weights (``loop``), every pass with a cache
and a state of its own.  A final RMS norm and a head.  Every size and every constant that may differ between models comes from config.json:

    {"architecture": "Lefilorn", "vocab": V, "width": W, "norm": {"eps": e}, "embedding": {"scale": s}, "streams": n,
     "loop": {"start": a, "stop": b, "times": n},
     "layers": [{"type": "parallel", "mixer": {"left": {"heads", "kv_heads", "dim", "vdim", "scale", "mask": {"size", "keep_first"},
                 "rot": {"base", "dims"}}, "right": {"heads", "dim", "vdim", "decay": [per head], "rot": {"base", "dims"}},
                 "left_scale", "right_scale"}, "mlp": null | {"kind": "dense", "ff": F}}]}

Without ``streams`` a layer is x += sublayer(norm(x)) twice.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Optional, Tuple

from .registry import register_architecture
from .specs import (BranchSumSpec, ConfigError, GatedAttentionSpec, GatedMLPSpec, LayerSpec, LinearAttentionSpec, ModelPlan, NoPositionSpec,
                    RMSNormSpec, RotaryHalvesSpec, RotaryPairsSpec, ScheduleEntry, StreamMixSpec)

# Positions enter float32 angles: every integer below 2^24 is exact there.
MAX_POSITIONS = 1 << 24


def _int(d, key: str, where: str, least: int = 1) -> int:
    v = d.get(key) if isinstance(d, dict) else None
    if isinstance(v, bool) or not isinstance(v, int) or v < least:
        raise ConfigError(f"{where}{key} must be an integer of at least {least}, found {v!r}")
    return v


def _number(d, key: str, where: str, positive: bool = True) -> float:
    v = d.get(key) if isinstance(d, dict) else None
    if isinstance(v, bool) or not isinstance(v, (int, float)) or (positive and not v > 0):
        raise ConfigError(f"{where}{key} must be a {'positive ' if positive else ''}number, found {v!r}")
    return float(v)


def _rot(m: dict, where: str, most: int) -> Optional[dict]:
    rot = m.get("rot")
    if rot is None:
        return None
    out = {"base": _number(rot, "base", where + "rot."), "dims": _int(rot, "dims", where + "rot.", least=0)}
    if out["dims"] % 2 or out["dims"] > most:
        raise ConfigError(f"{where}rot.dims must be even and at most {most}, found {out['dims']}")
    return out


def _with_rot(out: dict, m: dict, where: str) -> dict:
    rot = _rot(m, where, out["dim"])
    if rot is not None:
        out["rot"] = rot
    return out


def _left(m, where: str) -> dict:
    if not isinstance(m, dict):
        raise ConfigError(f"{where[:-1]} must be an object with the attention's sizes")
    out = {k: _int(m, k, where) for k in ("heads", "kv_heads", "dim", "vdim")}
    out["scale"] = _number(m, "scale", where, positive=False)
    if out["heads"] % out["kv_heads"]:
        raise ConfigError(f"{where}: {out['heads']} heads cannot share {out['kv_heads']} key/value heads evenly")
    if m.get("mask") is not None:
        mask = {"size": _int(m["mask"], "size", where + "mask.")}
        if m["mask"].get("keep_first") is not None:
            mask["keep_first"] = _int(m["mask"], "keep_first", where + "mask.", least=0)
        out["mask"] = mask
    return _with_rot(out, m, where)


def _right(m, where: str) -> dict:
    if not isinstance(m, dict):
        raise ConfigError(f"{where[:-1]} must be an object with the linear attention's sizes")
    out = {k: _int(m, k, where) for k in ("heads", "dim", "vdim")}
    decay = m.get("decay")
    if (not isinstance(decay, list) or len(decay) != out["heads"]
            or not all(isinstance(a, (int, float)) and not isinstance(a, bool) and a >= 0 for a in decay)):
        raise ConfigError(f"{where}decay must list one number (not negative) for each of the {out['heads']} heads, found {decay!r}")
    out["decay"] = [float(a) for a in decay]
    return _with_rot(out, m, where)


def _mlp(mlp, where: str) -> Optional[dict]:
    if mlp is None:
        return None
    if not isinstance(mlp, dict) or mlp.get("kind") != "dense":
        raise ConfigError(f"{where}kind must be \"dense\" (or mlp null), found {mlp!r}")
    return {"ff": _int(mlp, "ff", where), "kind": "dense"}


@dataclass(frozen=True)
class LefilornLayer:
    """One entry of ``layers``: ``kind`` and the checked ``mixer`` and ``mlp`` objects as config.json spells them."""
    kind: str
    mixer: dict = field(hash=False)
    mlp: Optional[dict] = field(default=None, hash=False)

    @classmethod
    def from_dict(cls, d: dict, i: int) -> "LefilornLayer":
        where = f"layers[{i}]."
        if not isinstance(d, dict) or "type" not in d:
            raise ConfigError(f"layers[{i}] needs a type")
        kind, m = d["type"], d.get("mixer")
        if kind != "parallel":
            raise ConfigError(f"{where}type must be \"parallel\", found {kind!r}")
        if not isinstance(m, dict):
            raise ConfigError(f"{where}mixer must be an object with left, right and their scales")
        mixer = {"left": _left(m.get("left"), where + "mixer.left."), "right": _right(m.get("right"), where + "mixer.right.")}
        for k in ("left_scale", "right_scale"):
            mixer[k] = _number(m, k, where + "mixer.", positive=False)
        return cls(kind, mixer, _mlp(d.get("mlp"), where + "mlp."))

    def to_dict(self) -> dict:
        return {"mixer": {k: dict(v) if isinstance(v, dict) else v for k, v in self.mixer.items()}, "mlp": self.mlp, "type": self.kind}


@dataclass(frozen=True)
class LefilornConfig:
    ARCHITECTURE = "Lefilorn"

    vocab: int
    width: int
    layers: Tuple[LefilornLayer, ...]
    norm_eps: float
    embedding_scale: float = 1.0
    streams: Optional[int] = None
    loop: Optional[Tuple[int, int, int]] = None       # (start, stop, times)

    @classmethod
    def from_dict(cls, d: dict) -> "LefilornConfig":
        missing = [k for k in ("vocab", "width", "layers", "norm") if d.get(k) is None]
        if missing:
            raise ConfigError("config.json lacks " + ", ".join(missing))
        if not isinstance(d["layers"], list) or not d["layers"]:
            raise ConfigError("layers must be a non-empty list")
        if not isinstance(d["norm"], dict):
            raise ConfigError("norm must be an object ({\"eps\": ...})")
        loop = d.get("loop")
        if loop is not None:
            a, b, n = (loop.get(k) for k in ("start", "stop", "times")) if isinstance(loop, dict) else (None,) * 3
            if not all(isinstance(v, int) and not isinstance(v, bool) for v in (a, b, n)) or not 0 <= a < b <= len(d["layers"]) or n < 1:
                raise ConfigError(f"loop needs 0 <= start < stop <= {len(d['layers'])} layers and times >= 1, found {loop!r}")
            loop = (a, b, n)
        emb = d.get("embedding")
        scale = 1.0 if not isinstance(emb, dict) or emb.get("scale") is None else _number(emb, "scale", "embedding.", positive=False)
        return cls(vocab=_int(d, "vocab", ""), width=_int(d, "width", ""), layers=tuple(LefilornLayer.from_dict(x, i) for i, x in enumerate(d["layers"])),
                   norm_eps=_number(d["norm"], "eps", "norm."), embedding_scale=scale,
                   streams=None if d.get("streams") is None else _int(d, "streams", ""), loop=loop)

    def to_dict(self) -> dict:
        d = {"architecture": self.ARCHITECTURE, "embedding": {"scale": self.embedding_scale}, "layers": [x.to_dict() for x in self.layers],
             "norm": {"eps": self.norm_eps}, "vocab": self.vocab, "width": self.width}
        if self.streams is not None:
            d["streams"] = self.streams
        if self.loop is not None:
            d["loop"] = {"start": self.loop[0], "stop": self.loop[1], "times": self.loop[2]}
        return d

    # ---------------------------------------------------------------- the plan

    def _mixer_spec(self, x: LefilornLayer, p: str) -> BranchSumSpec:
        W, eps, left, right = self.width, self.norm_eps, x.mixer["left"], x.mixer["right"]
        rot, mask = left.get("rot"), left.get("mask") or {}
        position = NoPositionSpec() if rot is None else RotaryPairsSpec(head_dim=left["dim"], dims=rot["dims"], base=rot["base"])
        attention = GatedAttentionSpec(hidden=W, n_heads=left["heads"], n_kv_heads=left["kv_heads"], head_dim=left["dim"], v_head_dim=left["vdim"],
                                       window=mask.get("size"), keep_first=mask.get("keep_first", 0), scale=left["scale"], position=position,
                                       prefix=p + "left.", norm_eps=eps, gate="g", bias=True, o_bias=False, qk_row_norm=("q.norm", "k.norm"))
        rot = right.get("rot")
        position = None if rot is None else RotaryHalvesSpec(head_dim=right["dim"], dims=rot["dims"], base=rot["base"])
        retention = LinearAttentionSpec(hidden=W, n_heads=right["heads"], head_dim=right["dim"], v_head_dim=right["vdim"], prefix=p + "right.",
                                        head_decay=tuple(right["decay"]), norm_over="head", norm_eps=eps, norm_name=None, gate_activation="silu",
                                        position=position, k_scale=right["dim"] ** -0.5)
        return BranchSumSpec(hidden=W, branches=(attention, retention), out_norms=None, norm_eps=eps,
                             scales=(x.mixer["left_scale"], x.mixer["right_scale"]))

    def plan(self) -> ModelPlan:
        W, eps, n = self.width, self.norm_eps, len(self.layers)

        def mix(p: str, there: bool = True) -> Optional[StreamMixSpec]:
            return StreamMixSpec(self.streams, p + "in", p + "out", p + "mix") if self.streams is not None and there else None
        layers, unused = [], []
        for i, x in enumerate(self.layers):
            p = f"l{i}."
            ff = None if x.mlp is None else GatedMLPSpec(W, x.mlp["ff"], p + "mlp.", activation="relu")
            layers.append(LayerSpec(mixer=self._mixer_spec(x, p + "mix."), mixer_norm=RMSNormSpec(W, eps, p + "norm1"), feed_forward=ff,
                                    feed_forward_norm=None if ff is None else RMSNormSpec(W, eps, p + "norm2"),
                                    arrangement="pre_norm" if self.streams is None else "streams",
                                    mixer_streams=mix(p + "hc1."), feed_forward_streams=mix(p + "hc2.", ff is not None)))
            if ff is None:                                   # a layer without a feed-forward may still store what would stand around it
                unused.extend(p + n for n in ("norm2", "hc2.in", "hc2.out", "hc2.mix"))
        order = list(range(n))
        if self.loop is not None:
            a, b, times = self.loop
            order = order[:a] + order[a:b] * times + order[b:]
        plan = ModelPlan(architecture=self.ARCHITECTURE, vocab_size=self.vocab, hidden_size=W, embedding="embed", layers=tuple(layers),
                         schedule=tuple(ScheduleEntry(i) for i in order), final_norm=RMSNormSpec(W, eps, "final.norm"), head="head",
                         max_positions=MAX_POSITIONS, ignorable_tensors=tuple(unused), embedding_scale=self.embedding_scale,
                         streams=self.streams)
        plan.validate()
        return plan


register_architecture(LefilornConfig.ARCHITECTURE, LefilornConfig)
