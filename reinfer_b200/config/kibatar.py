"""Typed configuration of the Kibatar architecture: a decoder whose layers are listed one by one in config.json, each with
latent attention or a recurrent `wkv` mixer and with a mixture of experts (or no feed-forward); a stretch of layers may run
several times in a row.

    {"architecture": "Kibatar", "vocab": V, "width": h, "norm": {"eps": e}, "logit_scale": c,
     "embedding": {"scale": s, "bigram": {"buckets": B, "mul_prev": m, "mul_cur": n}},
     "loop": {"start": a, "stop": b, "times": t},
     "layers": [{"type": "latent_attention",
                 "mixer": {"heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank", "scale",
                           "rot": {"base", "dims", "scaling": {"factor", "original", "fast", "slow"}}},
                 "mlp": null | {"kind": "moe", "expert": {"ff": F, "limit": L}, "shared": {"ff": S, "limit": M},
                                "router": {"experts": E, "top": k, "scale": r}}}
                | {"type": "wkv", "mixer": {"heads", "dim"}, "mlp": ...}, ...]}

`bigram`, `loop`, `scaling` and `shared` may be absent.  The rank of the wkv mixer's decay is read off the tensor
`l<i>.mix.w1` (or given as `decay_rank`); every other size and constant comes from the file.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Any, Dict, Mapping, Optional, Tuple

from .errors import InvalidValue, MissingKey

MIXER_TYPES = ("latent_attention", "wkv")
_LATENT_SIZES = ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank")
_SCALING = ("factor", "original", "fast", "slow")


def _int(d: Mapping[str, Any], key: str, where: str, least: int = 1) -> int:
    v = d.get(key)
    if v is None:
        raise MissingKey(f"{where}.{key}")
    if isinstance(v, bool) or not isinstance(v, int) or v < least:
        raise InvalidValue(f"{where}.{key}", f"expected an integer of at least {least}, got {v!r}")
    return int(v)


def _number(d: Mapping[str, Any], key: str, where: str, positive: bool = False) -> float:
    v = d.get(key)
    if v is None:
        raise MissingKey(f"{where}.{key}")
    if isinstance(v, bool) or not isinstance(v, (int, float)) or not math.isfinite(v) or (positive and v <= 0):
        raise InvalidValue(f"{where}.{key}", f"expected a {'positive' if positive else 'finite'} number, got {v!r}")
    return float(v)


def _section(d: Mapping[str, Any], key: str, where: str) -> Mapping[str, Any]:
    v = d.get(key)
    if v is None:
        raise MissingKey(f"{where}.{key}")
    if not isinstance(v, Mapping):
        raise InvalidValue(f"{where}.{key}", f"expected an object, got {v!r}")
    return v


def _parse_latent(m: Mapping[str, Any], where: str) -> dict:
    out: Dict[str, Any] = {k: _int(m, k, where) for k in _LATENT_SIZES}
    out["scale"] = _number(m, "scale", where)
    r, rw = _section(m, "rot", where), where + ".rot"
    dims = _int(r, "dims", rw)
    if dims % 2 or dims > out["rot_dim"]:
        raise InvalidValue(rw + ".dims", f"{dims} rotated dimensions of {out['rot_dim']}")
    scaling = None
    if r.get("scaling") is not None:
        s = _section(r, "scaling", rw)
        scaling = {k: _number(s, k, rw + ".scaling", positive=True) for k in _SCALING}
    out["rot"] = {"base": _number(r, "base", rw, positive=True), "dims": dims, "scaling": scaling}
    return out


def _parse_wkv(m: Mapping[str, Any], shapes, prefix: str, where: str) -> dict:
    rank = m.get("decay_rank")
    if rank is not None:
        rank = _int(m, "decay_rank", where)
    else:
        if shapes is None or prefix + "w1" not in shapes:
            raise MissingKey(f"{where}.decay_rank (or the tensor {prefix}w1)")
        rank = int(shapes[prefix + "w1"][0])
    return {"heads": _int(m, "heads", where), "dim": _int(m, "dim", where), "decay_rank": rank}


def _parse_mlp(mlp, where: str):
    if mlp is None:
        return None
    if not isinstance(mlp, Mapping) or mlp.get("kind") != "moe":
        raise InvalidValue(where + ".kind", f"expected 'moe', got {mlp!r}")
    r, rw = _section(mlp, "router", where), where + ".router"
    experts, top = _int(r, "experts", rw), _int(r, "top", rw)
    if top > experts:
        raise InvalidValue(rw + ".top", f"{top} of {experts} experts")

    def expert(key: str):
        s = _section(mlp, key, where)
        return {"ff": _int(s, "ff", f"{where}.{key}"), "limit": _number(s, "limit", f"{where}.{key}", positive=True)}

    return {"kind": "moe", "expert": expert("expert"), "shared": None if mlp.get("shared") is None else expert("shared"),
            "router": {"experts": experts, "top": top, "scale": _number(r, "scale", rw)}}


@dataclass(frozen=True)
class KibatarLayer:
    type: str
    mixer: Any                       # a plain dict of validated sizes and constants
    mlp: Any                         # None or {"kind": "moe", "expert", "shared" (or None), "router"}


@dataclass(frozen=True)
class KibatarConfig:
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    logit_scale: float
    layers: Tuple[KibatarLayer, ...]
    bigram: Optional[Tuple[int, int, int]] = None      # (buckets, mul_prev, mul_cur)
    loop: Optional[Tuple[int, int, int]] = None        # (start, stop, times)
    eos_token_ids: Tuple[int, ...] = ()
    architecture: str = "Kibatar"

    default_eos_ids = ()
    reads_tensor_shapes = True       # load_config hands from_dict the checkpoint's tensor shapes

    # names the serving code asks of any configuration
    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    @classmethod
    def from_dict(cls, d: Mapping[str, Any], shapes: Optional[Mapping[str, Tuple[int, ...]]] = None) -> "KibatarConfig":
        vocab, width = _int(d, "vocab", "config"), _int(d, "width", "config")
        eps = _number(_section(d, "norm", "config"), "eps", "norm")
        if eps < 0:
            raise InvalidValue("norm.eps", "must be >= 0")
        emb = _section(d, "embedding", "config")
        bigram = None
        if emb.get("bigram") is not None:
            b, bw = _section(emb, "bigram", "embedding"), "embedding.bigram"
            bigram = (_int(b, "buckets", bw), _int(b, "mul_prev", bw, 0), _int(b, "mul_cur", bw, 0))
        raw_layers = d.get("layers")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise MissingKey("layers")
        layers = []
        for i, rl in enumerate(raw_layers):
            where = f"layers[{i}]"
            if not isinstance(rl, Mapping) or rl.get("type") not in MIXER_TYPES:
                raise InvalidValue(where + ".type", f"expected one of {MIXER_TYPES}, got {rl.get('type') if isinstance(rl, Mapping) else rl!r}")
            m, mw = _section(rl, "mixer", where), where + ".mixer"
            mixer = _parse_wkv(m, shapes, f"l{i}.mix.", mw) if rl["type"] == "wkv" else _parse_latent(m, mw)
            layers.append(KibatarLayer(rl["type"], mixer, _parse_mlp(rl.get("mlp"), where + ".mlp")))
        loop = None
        if d.get("loop") is not None:
            lp = _section(d, "loop", "config")
            loop = (_int(lp, "start", "loop", 0), _int(lp, "stop", "loop"), _int(lp, "times", "loop"))
            if not loop[0] < loop[1] <= len(layers):
                raise InvalidValue("loop", f"layers {loop[0]} to {loop[1]} of {len(layers)}")
        eos = d.get("eos_token_id")
        eos_ids = () if eos is None else ((int(eos),) if isinstance(eos, int) else tuple(int(e) for e in eos))
        return cls(vocab=vocab, width=width, norm_eps=eps, embedding_scale=_number(emb, "scale", "embedding"),
                   logit_scale=_number(d, "logit_scale", "config"), layers=tuple(layers), bigram=bigram, loop=loop, eos_token_ids=eos_ids)

    def to_dict(self) -> dict:
        layers = []
        for l in self.layers:
            if l.type == "wkv":
                mixer = dict(l.mixer)
            else:
                rot = {k: v for k, v in l.mixer["rot"].items() if v is not None}
                mixer = {**{k: l.mixer[k] for k in _LATENT_SIZES + ("scale",)}, "rot": rot}
            mlp = None if l.mlp is None else {k: dict(v) if isinstance(v, Mapping) else v for k, v in l.mlp.items() if v is not None}
            layers.append({"type": l.type, "mixer": mixer, "mlp": mlp})
        emb: Dict[str, Any] = {"scale": self.embedding_scale}
        if self.bigram is not None:
            emb["bigram"] = dict(zip(("buckets", "mul_prev", "mul_cur"), self.bigram))
        out: Dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
                               "norm": {"eps": self.norm_eps}, "embedding": emb, "logit_scale": self.logit_scale, "layers": layers}
        if self.loop is not None:
            out["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        if self.eos_token_ids:
            out["eos_token_id"] = list(self.eos_token_ids)
        return out
