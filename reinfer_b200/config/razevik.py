"""Typed configuration of the Razevik architecture: a decoder whose layers are listed one by one in config.json, all
with latent attention without positions, and each with a dense or expert-mixture feed-forward (or none).

    {"architecture": "Razevik", "vocab": V, "width": h, "max_positions": P, "norm": {"eps": e},
     "residual_mult": m, "logit_softcap": c, "token_side": {"dim": d},
     "layers": [{"type": "latent_attention",
                 "mixer": {"heads", "dim", "vdim", "q_rank", "kv_rank", "scale", "kv_from": j},
                 "mlp": null | {"kind": "dense", "ff": F}
                             | {"kind": "moe", "expert": {"ff": F}, "shared": {"ff": S},
                                "router": {"experts": E, "top": k, "groups": {"count": g, "keep": n}}}}, ...]}

`kv_from` (the layer whose cached latent this one reads), `shared`, `groups`, `logit_softcap` and `token_side` may be
absent (a latent of its own, no shared expert, one free choice among all experts, plain logits, no token rows).  Every
size and constant comes from the file; nothing is read off tensor shapes.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Any, Dict, Mapping, Optional, Tuple

from .errors import InvalidValue, MissingKey

MIXER_TYPES = ("latent_attention",)
_SIZES = ("heads", "dim", "vdim", "q_rank", "kv_rank")


def _pos_int(d: Mapping[str, Any], key: str, where: str) -> int:
    v = d.get(key)
    if v is None:
        raise MissingKey(f"{where}.{key}")
    if isinstance(v, bool) or not isinstance(v, int) or v <= 0:
        raise InvalidValue(f"{where}.{key}", f"expected a positive integer, got {v!r}")
    return int(v)


def _number(d: Mapping[str, Any], key: str, where: str) -> float:
    v = d.get(key)
    if v is None:
        raise MissingKey(f"{where}.{key}")
    if isinstance(v, bool) or not isinstance(v, (int, float)) or not math.isfinite(v):
        raise InvalidValue(f"{where}.{key}", f"expected a finite number, got {v!r}")
    return float(v)


def _section(d: Mapping[str, Any], key: str, where: str) -> Mapping[str, Any]:
    v = d.get(key)
    if v is None:
        raise MissingKey(f"{where}.{key}")
    if not isinstance(v, Mapping):
        raise InvalidValue(f"{where}.{key}", f"expected an object, got {v!r}")
    return v


def _parse_mixer(m: Mapping[str, Any], where: str) -> dict:
    out: Dict[str, Any] = {k: _pos_int(m, k, where) for k in _SIZES}
    out["scale"] = _number(m, "scale", where)
    src = m.get("kv_from")
    if src is not None and (isinstance(src, bool) or not isinstance(src, int)):
        raise InvalidValue(where + ".kv_from", f"expected a layer's number, got {src!r}")
    out["kv_from"] = src
    return out


def _parse_mlp(mlp, where: str):
    if mlp is None:
        return None
    if not isinstance(mlp, Mapping) or mlp.get("kind") not in ("dense", "moe"):
        raise InvalidValue(where + ".kind", f"expected 'dense' or 'moe', got {mlp!r}")
    if mlp["kind"] == "dense":
        return {"kind": "dense", "ff": _pos_int(mlp, "ff", where)}
    r, rw = _section(mlp, "router", where), where + ".router"
    experts, top = _pos_int(r, "experts", rw), _pos_int(r, "top", rw)
    groups = None
    if r.get("groups") is not None:
        g = _section(r, "groups", rw)
        groups = (_pos_int(g, "count", rw + ".groups"), _pos_int(g, "keep", rw + ".groups"))
        if experts % groups[0]:
            raise InvalidValue(rw + ".groups.count", f"{experts} experts do not form {groups[0]} equal groups")
        if groups[1] > groups[0]:
            raise InvalidValue(rw + ".groups.keep", f"{groups[1]} of {groups[0]} groups")
    allowed = experts if groups is None else experts // groups[0] * groups[1]
    if top > allowed:
        raise InvalidValue(rw + ".top", f"{top} of {allowed} experts that a token may choose")
    shared = None
    if mlp.get("shared") is not None:
        shared = _pos_int(_section(mlp, "shared", where), "ff", where + ".shared")
    return {"kind": "moe", "ff": _pos_int(_section(mlp, "expert", where), "ff", where + ".expert"), "experts": experts,
            "top": top, "groups": groups, "shared": shared}


@dataclass(frozen=True)
class RazevikLayer:
    type: str
    mixer: Any                       # a plain dict of validated sizes and constants, `kv_from` included
    mlp: Any                         # None, {"kind": "dense", "ff"} or {"kind": "moe", "ff", "experts", "top", "groups", "shared"}


@dataclass(frozen=True)
class RazevikConfig:
    vocab: int
    width: int
    max_positions: int
    norm_eps: float
    residual_mult: float
    layers: Tuple[RazevikLayer, ...]
    logit_softcap: Optional[float] = None
    side_dim: Optional[int] = None
    eos_token_ids: Tuple[int, ...] = ()
    architecture: str = "Razevik"

    default_eos_ids = ()

    # names the serving code asks of any configuration
    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "RazevikConfig":
        vocab, width = _pos_int(d, "vocab", "config"), _pos_int(d, "width", "config")
        max_positions = _pos_int(d, "max_positions", "config")
        eps = _number(_section(d, "norm", "config"), "eps", "norm")
        if eps < 0:
            raise InvalidValue("norm.eps", "must be >= 0")
        mult = _number(d, "residual_mult", "config")
        cap = None
        if d.get("logit_softcap") is not None:
            cap = _number(d, "logit_softcap", "config")
            if cap <= 0:
                raise InvalidValue("logit_softcap", "must be positive")
        side = None
        if d.get("token_side") is not None:
            side = _pos_int(_section(d, "token_side", "config"), "dim", "token_side")
        raw_layers = d.get("layers")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise MissingKey("layers")
        layers = []
        for i, rl in enumerate(raw_layers):
            where = f"layers[{i}]"
            if not isinstance(rl, Mapping) or rl.get("type") not in MIXER_TYPES:
                raise InvalidValue(where + ".type", f"expected one of {MIXER_TYPES}, got {rl.get('type') if isinstance(rl, Mapping) else rl!r}")
            layers.append(RazevikLayer(rl["type"], _parse_mixer(_section(rl, "mixer", where), where + ".mixer"),
                                       _parse_mlp(rl.get("mlp"), where + ".mlp")))
        for i, l in enumerate(layers):
            src = l.mixer["kv_from"]
            if src is None:
                continue
            where = f"layers[{i}].mixer.kv_from"
            if not 0 <= src < i:
                raise InvalidValue(where, f"layer {i} can read the latent of an earlier layer only, got {src}")
            s = layers[src].mixer
            if s["kv_from"] is not None:
                raise InvalidValue(where, f"layer {src} has no latent of its own")
            if s["kv_rank"] != l.mixer["kv_rank"]:
                raise InvalidValue(where, f"layers {src} and {i} differ in 'kv_rank'")
        eos = d.get("eos_token_id")
        eos_ids = () if eos is None else ((int(eos),) if isinstance(eos, int) else tuple(int(e) for e in eos))
        return cls(vocab=vocab, width=width, max_positions=max_positions, norm_eps=eps, residual_mult=mult, layers=tuple(layers),
                   logit_softcap=cap, side_dim=side, eos_token_ids=eos_ids)

    def to_dict(self) -> dict:
        layers = []
        for l in self.layers:
            mixer = {k: l.mixer[k] for k in _SIZES + ("scale",)}
            if l.mixer["kv_from"] is not None:
                mixer["kv_from"] = l.mixer["kv_from"]
            mlp = l.mlp
            if mlp is not None and mlp["kind"] == "dense":
                mlp = {"kind": "dense", "ff": mlp["ff"]}
            elif mlp is not None:
                router: Dict[str, Any] = {"experts": mlp["experts"], "top": mlp["top"]}
                if mlp["groups"] is not None:
                    router["groups"] = {"count": mlp["groups"][0], "keep": mlp["groups"][1]}
                out_mlp: Dict[str, Any] = {"kind": "moe", "expert": {"ff": mlp["ff"]}, "router": router}
                if mlp["shared"] is not None:
                    out_mlp["shared"] = {"ff": mlp["shared"]}
                mlp = out_mlp
            layers.append({"type": l.type, "mixer": mixer, "mlp": mlp})
        out: Dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
                               "max_positions": self.max_positions, "norm": {"eps": self.norm_eps},
                               "residual_mult": self.residual_mult, "layers": layers}
        if self.logit_softcap is not None:
            out["logit_softcap"] = self.logit_softcap
        if self.side_dim is not None:
            out["token_side"] = {"dim": self.side_dim}
        if self.eos_token_ids:
            out["eos_token_id"] = list(self.eos_token_ids)
        return out
